"""The Gatarax decoder in the engine against the plain restatement (`plain_gatarax`): each mechanism's kernels alone,
then whole models: prompts whole, token by token, in portions down to two tokens, unequal batches, slots and pages used
again, keys at the edges of windows and of pages, far tokens, the first tokens of a sequence, long decoding, and greedy
generation through `Model.generate`."""
import math

import pytest
import torch

import gatarax_models as gm
import plain_gatarax as pg
from conftest import random_tokens, rel_err
from test_belizen_gpu import Streams, _Scratch, _run
from test_redodra_gpu import _drive, d, i32, make_ctx

# Worst row's max |a - b| / max |b| against the plain model in float64.  float32 runs: a kernel fault shows far above
# 1e-4.  bfloat16 runs keep bfloat16 activations between the kernels of a sublayer (the stream, the states, the norms,
# the router and the scores stay float32): rounding alone reaches 1e-2; a key too many or too few, a lost state, a missing
# sink or a wrong expert costs 0.2 and more.
TOL = {"float32": 1e-4, "bfloat16": 4e-2}

pytestmark = pytest.mark.gpu

DEV = "cuda"
F32, BF16 = torch.float32, torch.bfloat16
PART_TOL = {F32: 3e-5, BF16: 3e-2}


def _cache(part, dtype, n_slots=2, max_tokens=1024):
    from rust_inference_b200.cache.sequence_cache import SequenceCache
    return SequenceCache([part.cache_request()], max_tokens=max_tokens, max_seq_len=512, dtype=dtype, device=DEV, n_slots=n_slots)


def _workspace():
    from rust_inference_b200.engine.context import Workspace
    return Workspace(DEV)


LEFT = gm.left(heads=1, kv=1, dim=8, vdim=8, scale=1.0, conv=1, size=1)
RIGHT = gm.right(heads=1, kv=1, dim=8, vdim=8, conv=1)


def _part(kind, m, dtype, width, seed, eps=1e-5, edit=None, pin=False, ranks=None, hot=1.0):
    """One part of the library as the model's builder makes it for a one-layer model, holding random tensors; the same
    tensors in float64 for the plain functions, and the tensors' prefix.  kind: "left", "right", "parallel", "lightning" or
    "mlp"."""
    from rust_inference_b200.config.registry import get_architecture
    from rust_inference_b200.parts.registry import lookup
    mlp = m if kind == "mlp" else None
    if kind == "lightning":
        layer = {"type": "lightning", "mixer": m, "mlp": None}
    else:
        layer = gm.parallel(m if kind == "left" else m["left"] if kind == "parallel" else LEFT,
                            m if kind == "right" else m["right"] if kind == "parallel" else RIGHT, mlp)
    cfg = gm.model(vocab=10, width=width, eps=eps, taps=1, scale=1.0, logit_scale=1.0, layers=[layer])
    W = pg.random_weights(cfg, seed, hot=hot, ranks=ranks)
    if pin:
        gm.pin_routing(cfg, W)
    W = {k: v.float() for k, v in W.items()}
    prefix = {"left": "l0.mix.left.", "right": "l0.mix.right.", "mlp": "l0.mlp."}.get(kind, "l0.mix.")
    if edit is not None:
        edit(W, prefix)
    arch = get_architecture("Gatarax")
    spec = arch.build_spec(arch.parse_config(cfg, shapes={k: tuple(v.shape) for k, v in W.items()})).layers[0]
    ps = spec.parts["feed_forward" if kind == "mlp" else "mixer"]
    if kind in ("left", "right"):
        ps = ps.params["members"][0 if kind == "left" else 1][0]
    part = lookup("feed_forward" if kind == "mlp" else "mixer", ps.kind)(hidden_size=width, dtype=dtype, device=DEV, **ps.params)
    part.set_tensors({local: d(W[prefix + local], F32 if ts.role == "vector" else dtype) for local, ts in part.tensor_specs().items()})
    part.prepare(2048)
    return part, {k: v.double() for k, v in W.items()}, prefix


# ---------------------------------------------------------------------------------------------------
# kernels alone
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width,taps,two,normed", [(96, 4, True, True), (72, 1, True, True), (130, 2, False, True), (64, 3, True, False),
                                                   (1030, 5, True, True), (4096, 4, True, True), (40, 7, False, False)])
def test_input_convolutions(dtype, width, taps, two, normed):
    """h = norm(x) of the float32 stream, h + conv_a(h) and h + conv_b(h) in one kernel, over three sequences of a packed
    step (one of a single token, one shorter than the filter, one of 600: several tokens per block), continued by portions and
    by single tokens, in slots that held other sequences."""
    from rust_inference_b200.kernels import ops
    g = torch.Generator().manual_seed(width + taps)
    w = 1.0 + 0.3 * torch.randn(width, generator=g) if normed else None
    fa, fb = (torch.randn(width, taps, generator=g) / math.sqrt(taps) for _ in range(2))
    carried = torch.full((4, taps - 1, width), 7.0, device=DEV)
    slots = [2, 0, 3]
    carried[slots] = 0.0
    total = [606, 9, 23]
    xs = [torch.randn(n, width, generator=g) * 3 for n in total]
    want = []
    for x in xs:
        h = pg.unit_rms(x.double(), 1e-5) * w.double() if normed else x.double()
        want.append((pg.input_conv(h, fa.double()), pg.input_conv(h, fb.double())))
    at = [0, 0, 0]
    got = [([], []), ([], []), ([], [])]
    for counts in ([600, 1, 2], [2, 2, 3], [1, 1, 1], [3, 3, 16], [0, 1, 0], [0, 1, 1]):
        live = [i for i in range(3) if counts[i]]
        n = sum(counts)
        x = d(torch.cat([xs[i][at[i]:at[i] + counts[i]] for i in live]))
        cu = [0]
        for i in live:
            cu.append(cu[-1] + counts[i])
        seq = [b for b, i in enumerate(live) for _ in range(counts[i])]
        a = torch.empty(n, width, dtype=dtype, device=DEV)
        b = torch.empty(n, width, dtype=dtype, device=DEV) if two else None
        ops.input_conv(x, d(w) if normed else None, 1e-5, d(fa.t().contiguous()), d(fb.t().contiguous()) if two else None, carried, a, b,
                       i32(cu), i32(seq), i32([slots[i] for i in live]), n_seqs=len(live), longest_run=max(counts))
        for k, i in enumerate(live):
            got[i][0].append(a[cu[k]:cu[k + 1]].float().cpu())
            if two:
                got[i][1].append(b[cu[k]:cu[k + 1]].float().cpu())
            at[i] += counts[i]
    assert at == total
    for i in range(3):
        for side in range(2 if two else 1):
            assert rel_err(torch.cat(got[i][side]), want[i][side]) < (1e-5 if dtype == F32 else 6e-3), (i, side)
    assert taps == 1 or float(carried[1].min()) == 7.0               # nobody else's slot was touched


@pytest.mark.parametrize("width,taps", [(40, 4), (36, 2), (33, 3), (64, 6)])
def test_input_convolutions_of_a_very_long_step(width, taps):
    """A step of more than 4,096 tokens takes eight tokens per block: two sequences whose border lies inside a block."""
    from rust_inference_b200.kernels import ops
    g = torch.Generator().manual_seed(width)
    w = 1.0 + 0.3 * torch.randn(width, generator=g)
    fa, fb = (torch.randn(width, taps, generator=g) / math.sqrt(taps) for _ in range(2))
    counts = [2803, 1402]
    xs = [torch.randn(n, width, generator=g) for n in counts]
    carried = torch.zeros(2, taps - 1, width, device=DEV)
    a, b = (torch.empty(sum(counts), width, device=DEV) for _ in range(2))
    seq = torch.repeat_interleave(torch.arange(2), torch.tensor(counts)).tolist()
    ops.input_conv(d(torch.cat(xs)), d(w), 1e-5, d(fa.t().contiguous()), d(fb.t().contiguous()), carried, a, b, i32([0, 2803, 4205]), i32(seq),
                   i32([1, 0]), n_seqs=2, longest_run=2803)
    for k, (x, slot) in enumerate(zip(xs, (1, 0))):
        h = pg.unit_rms(x.double(), 1e-5) * w.double()
        part = slice(0, 2803) if k == 0 else slice(2803, 4205)
        assert rel_err(a[part], pg.input_conv(h, fa.double())) < 1e-5
        assert rel_err(b[part], pg.input_conv(h, fb.double())) < 1e-5
        assert rel_err(carried[slot], h[-(taps - 1):]) < 1e-5


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("n,width,ff", [(1, 72, 40), (5, 128, 200), (130, 128, 264), (600, 256, 520), (2100, 512, 1024), (9, 100, 36)])
def test_relu_squared_in_the_product_s_epilogue(dtype, n, width, ff):
    """max(x W^T, 0)^2 as one kernel: few and many tokens (every form of the tensor-core kernel), sizes it refuses."""
    from rust_inference_b200.kernels import linear, ops
    g = torch.Generator().manual_seed(n + ff)
    x = torch.randn(n, width, generator=g).to(dtype)
    w = (torch.randn(ff, width, generator=g) * (2.0 / math.sqrt(width))).to(dtype)
    out = torch.empty(n, ff, dtype=dtype, device=DEV)
    linear.activated(d(x), linear.Weight(d(w)), out, None, torch.tensor(ops.RELU_SQUARED_FORM, device=DEV))
    assert rel_err(out, torch.relu(x.double() @ w.double().T) ** 2) < (1e-5 if dtype == F32 else 1e-2)
    assert float(out.float().min()) == 0.0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("n,width,cols,total", [(1, 72, 40, 60), (7, 128, 200, 264), (130, 128, 100, 264), (600, 256, 300, 520),
                                                (2100, 512, 768, 1024), (9, 100, 36, 36), (33, 64, 0, 24)])
def test_silu_of_the_first_columns_in_the_product_s_epilogue(dtype, n, width, cols, total):
    """x W^T in float32 with silu on the first columns only, in every form of the contraction."""
    from rust_inference_b200.kernels import linear
    g = torch.Generator().manual_seed(n + cols)
    x = torch.randn(n, width, generator=g).to(dtype)
    w = (torch.randn(total, width, generator=g) * (3.0 / math.sqrt(width))).to(dtype)
    out = torch.empty(n, total, dtype=F32, device=DEV)
    linear.logits(d(x), linear.Weight(d(w)), out, None, silu_cols=torch.tensor([float(cols)], device=DEV))
    z = x.double() @ w.double().T
    z[:, :cols] = pg.silu(z[:, :cols])
    assert rel_err(out, z) < 1e-5


def test_router_ranks_groups_by_their_best_score():
    """Ids and weights of the routing kernel against the plain router, with the router's rows in one block per token and
    cut over several; without a correction."""
    from rust_inference_b200.kernels import ops
    for n, width, experts, top, count, keep in ((1, 72, 6, 2, 3, 2), (9, 128, 16, 5, 8, 3), (40, 256, 72, 8, 8, 2), (700, 100, 32, 6, 4, 4),
                                                (3000, 64, 8, 2, 8, 2), (5, 64, 1, 1, 1, 1), (17, 64, 10, 4, 5, 2)):
        g = torch.Generator().manual_seed(n)
        x = torch.randn(n, width, generator=g)
        router = torch.randn(experts, width, generator=g) / math.sqrt(width) * 2
        ids, weights = pg.route(x.double(), router.double(), top, count, keep)
        sums = torch.empty(n, experts + 1, dtype=torch.float32, device=DEV)
        tickets = torch.zeros(n, dtype=torch.int32, device=DEV)
        for split in ((1, 2, 5) if n < 296 else (1,)):
            got_ids = torch.empty(n, top, dtype=torch.int32, device=DEV)
            got_w = torch.empty(n, top, dtype=torch.float32, device=DEV)
            ops.moe_route(d(x), d(router), None, got_ids, got_w, top=top, groups=count, keep=keep, softmax=True, normalise=False,
                          group_max=True, split=split, split_sums=sums, split_count=tickets)
            assert torch.equal(got_ids.cpu().long(), ids), (n, split)
            assert torch.allclose(got_w.cpu().double(), weights, rtol=2e-5, atol=1e-7), (n, split)


@pytest.mark.parametrize("out_dtype", [F32, BF16])
@pytest.mark.parametrize("groups,size,w_len", [(4, 24, 24), (1, 72, 72), (2, 640, 640), (1, 1030, 1030)])
def test_norm_with_a_sigmoid_gate(out_dtype, groups, size, w_len):
    from rust_inference_b200.kernels import ops
    g = torch.Generator().manual_seed(groups * size)
    n, col = 9, 5
    x = torch.randn(n, groups * size, generator=g) * 3
    gate = torch.randn(n, col + groups * size + 3, generator=g) * 2
    w = 1 + 0.3 * torch.randn(w_len, generator=g)
    want = (pg.unit_rms(x.double().view(n, groups, size), 1e-5) * w.double().repeat(groups * size // w_len).view(groups, size)).reshape(n, -1)
    want = want * torch.sigmoid(gate[:, col:col + groups * size].double())
    out = torch.empty(n, groups * size, dtype=out_dtype, device=DEV)
    ops.gated_group_norm(d(x), d(gate), col, d(w), out, groups=groups, group_size=size, gate_first=False, gate_act="sigmoid", eps=1e-5)
    assert rel_err(out, want) < (3e-6 if out_dtype == F32 else 6e-3)


# ---------------------------------------------------------------------------------------------------
# parts alone, outside an engine
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,kv,dim,vdim,conv,ranks", [(4, 2, 16, 24, 3, (5, 3)), (1, 1, 40, 72, 1, (1, 1)), (6, 2, 8, 8, 5, (16, 8)),
                                                          (4, 4, 64, 128, 4, (24, 40)), (2, 1, 128, 64, 2, (64, 7)),
                                                          (3, 3, 20, 130, 4, (2, 130)), (2, 2, 256, 32, 4, (9, 32)), (2, 1, 9, 7, 2, (3, 4))])
def test_delta_rule_with_channel_decays(dtype, heads, kv, dim, vdim, conv, ranks):
    """The delta rule as a whole prompt (its low-rank maps as products), in portions of up to 16 tokens (the maps formed by the
    preparing kernel), token by token and in a slot another sequence has used."""
    width, n = 96, 150
    m = gm.right(heads=heads, kv=kv, dim=dim, vdim=vdim, conv=conv)
    part, W, p = _part("right", m, dtype, width, seed=dim + vdim, hot=1.5, ranks=lambda i: ranks)
    x = torch.randn(n, width, generator=torch.Generator().manual_seed(conv)).to(dtype)
    want = pg.delta_rule(x.double(), W, p, m, 1e-5)
    cache, ws = _cache(part, dtype), _workspace()
    for portions in ([n], [1], [2], [70, 1, 1, 3, 33, 16, 17, 2], [3, 1]):
        assert rel_err(_drive(part, cache, x, portions, dtype, ws), want) < PART_TOL[dtype], portions


@pytest.mark.parametrize("heads,kv,dim,vdim,conv,ranks", [(4, 2, 16, 24, 3, (5, 3)), (1, 1, 40, 72, 1, (1, 1)), (6, 2, 8, 8, 5, (16, 8)),
                                                          (2, 1, 128, 64, 2, (64, 7)), (3, 3, 9, 7, 4, (3, 4)), (5, 5, 48, 200, 4, (9, 32)),
                                                          (2, 2, 256, 32, 4, (8, 8))])
def test_delta_rule_of_a_long_prompt(heads, kv, dim, vdim, conv, ranks):
    """Steps of 512 tokens and more prepare several tokens per block and keep the scan's blocks apart: a prompt of 700 tokens
    whole, cut so that the second portion begins inside a block's tokens, and two prompts in one step whose border lies inside
    one, each against the plain result."""
    width, n = 96, 700
    m = gm.right(heads=heads, kv=kv, dim=dim, vdim=vdim, conv=conv)
    part, W, p = _part("right", m, F32, width, seed=dim + vdim, hot=1.5, ranks=lambda i: ranks)
    x = torch.randn(n, width, generator=torch.Generator().manual_seed(conv))
    want = pg.delta_rule(x.double(), W, p, m, 1e-5)
    from rust_inference_b200.cache.sequence_cache import SequenceCache
    cache = SequenceCache([part.cache_request()], max_tokens=4096, max_seq_len=1024, dtype=F32, device=DEV, n_slots=3)
    ws = _workspace()
    for portions in ([n], [533, 1, 3, 163]):
        assert rel_err(_drive(part, cache, x, portions, F32, ws), want) < 5e-5, portions
    slots = [cache.alloc_slot(), cache.alloc_slot()]
    counts = [421, 3]
    out = torch.zeros(sum(counts) + 200, width, device=DEV)
    third = cache.alloc_slot()
    ctx = make_ctx(cache, slots + [third], [0, 0, 0], counts + [200], F32, ws)
    part.forward(d(torch.cat([x[:421], x[:3], x[:200]])), out, ctx, cache.layer(0), True)
    for first, count in ((0, 421), (421, 3), (424, 200)):
        assert rel_err(out[first:first + count], want[:count]) < 5e-5, count


@pytest.mark.parametrize("heads,vdim,state,groups,conv,ng", [(3, 16, 8, 1, 4, 1), (4, 8, 24, 2, 2, 4), (2, 130, 20, 2, 5, 1), (6, 12, 20, 3, 1, 9)])
def test_state_space_of_a_long_prompt(heads, vdim, state, groups, conv, ng):
    """The state space's preparing kernel shares the path of several tokens per block, with a bias and without unit vectors."""
    import plain_redodra
    import redodra_models
    from test_redodra_gpu import _mixer
    width, n = 80, 640
    m = redodra_models.ssm(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=ng)
    part, W, p = _mixer("ssm", m, F32, width, seed=state + vdim, hot=1.5)
    x = torch.randn(n, width, generator=torch.Generator().manual_seed(conv))
    want = plain_redodra.state_space(x.double(), W, p, m, 1e-5)
    from rust_inference_b200.cache.sequence_cache import SequenceCache
    cache = SequenceCache([part.cache_request()], max_tokens=2048, max_seq_len=1024, dtype=F32, device=DEV, n_slots=2)
    for portions in ([n], [517, 2, 121]):
        assert rel_err(_drive(part, cache, x, portions, F32, _workspace()), want) < 5e-5, portions


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_decays_differ_by_key_channel(dtype):
    """Half of the key channels forget at once and half never: what is written along a forgotten channel is gone a token later,
    what is written along a kept one is still there 300 tokens later.  With the channels exchanged the results exchange."""
    width, n, dim = 64, 320, 32
    m = gm.right(heads=2, kv=2, dim=dim, vdim=16, conv=1)
    x = (torch.randn(n, width, generator=torch.Generator().manual_seed(3)) * 0.5).to(dtype)
    loud = x.clone()
    loud[4] = loud[4] * 16

    def late(forgotten):
        def edit(W, p):
            W[p + "a2"].zero_()
            W[p + "A_log"].fill_(0.0)
            bias = torch.full((2, dim), -30.0)
            bias[:, forgotten] = 30.0
            W[p + "dt_bias"] = bias.reshape(-1)
            for name in ("q", "k"):                               # keys and queries live on the first half of the channels
                W[p + name].view(2, dim, width)[:, dim // 2:] = 0.0
            W[p + "b"].fill_(0.0)
            W[p + "v"][:, :] = W[p + "v"][:, :] * 0.3
        part, W, p = _part("right", m, dtype, width, seed=8, edit=edit)
        cache, ws = _cache(part, dtype), _workspace()
        out = []
        for t in (x, loud):
            want = pg.delta_rule(t.double(), W, p, m, 1e-5)
            for portions in ([n], [200, 1]):
                assert rel_err(_drive(part, cache, t, portions, dtype, ws), want) < (1e-4 if dtype == F32 else 4e-2)
            out.append(want)
        return float((out[0][5:15] - out[1][5:15]).abs().max() / out[0][5:15].abs().max())
    assert late(slice(0, dim // 2)) < 1e-6                       # the channels in use forget: no trace of token 4
    assert late(slice(dim // 2, dim)) > 0.05                     # only the unused ones do


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,dim,vdim,decay", [(3, 24, 40, (0.3, 0.99, 1.0)), (1, 72, 33, (0.9,)), (2, 8, 16, (0.0, 0.999)),
                                                  (4, 64, 64, (0.5, 0.8, 0.97, 0.999)), (2, 130, 100, (0.95, 0.6)), (5, 6, 9, (0.9,) * 5)])
def test_fixed_decay_attention_alone(dtype, heads, dim, vdim, decay):
    """The mixer over one sequence whole (long runs in pieces side by side), in portions, token by token, in a used slot."""
    width, n = 96, 300
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}
    part, W, p = _part("lightning", m, dtype, width, seed=dim, hot=1.2)
    x = (torch.randn(n, width, generator=torch.Generator().manual_seed(vdim)) * 0.7).to(dtype)
    want = pg.lightning(x.double(), W, p, m, 1e-5)
    cache, ws = _cache(part, dtype), _workspace()
    for portions in ([n], [140, 64, 5, 2, 1], [2], [129, 1]):
        assert rel_err(_drive(part, cache, x, portions, dtype, ws), want) < PART_TOL[dtype], portions


@pytest.mark.parametrize("kind", ["right", "lightning"])
def test_a_state_remembers_a_far_token(kind):
    """With decays of almost 1 one large early input stays in the state: 300 tokens later the output still differs by far more
    than rounding, the library agrees with the plain result on both, also token by token, and the two sequences as one batch
    equal each alone."""
    width, n = 64, 330
    if kind == "right":
        m, plain = gm.right(heads=2, kv=1, dim=32, vdim=16, conv=2), pg.delta_rule
    else:
        m, plain = {"heads": 2, "dim": 32, "vdim": 16, "decay": [0.9999, 0.9995]}, pg.lightning

    def slow(W, p):
        if kind == "right":
            W[p + "A_log"].fill_(-9.0)
            W[p + "dt_bias"].fill_(-1.0)
    part, W, p = _part(kind, m, F32, width, seed=5, edit=slow)
    a = torch.randn(n, width, generator=torch.Generator().manual_seed(9)) * 0.5
    b = a.clone()
    b[4] = b[4] * 8.0
    wa, wb = plain(a.double(), W, p, m, 1e-5), plain(b.double(), W, p, m, 1e-5)
    assert float((wa[-1] - wb[-1]).abs().max()) > 1e-2 * float(wa[-1].abs().max())
    cache, ws = _cache(part, F32, n_slots=3, max_tokens=2048), _workspace()
    for x, want in ((a, wa), (b, wb)):
        assert rel_err(_drive(part, cache, x, [n], F32, ws), want) < 1e-4
        assert rel_err(_drive(part, cache, x, [40, 1], F32, ws), want) < 1e-4
    slots = [cache.alloc_slot(), cache.alloc_slot()]
    got = [torch.zeros(n, width, device=DEV), torch.zeros(n, width, device=DEV)]
    at = [37, 5]
    out = torch.zeros(sum(at), width, device=DEV)
    part.forward(d(torch.cat([a[:37], b[:5]])), out, make_ctx(cache, slots, [0, 0], at, F32, ws), cache.layer(0), True)
    got[0][:37], got[1][:5] = out[:37], out[37:]
    for s, k in zip(slots, at):
        cache.commit(s, k)
    while min(at) < n:
        live = [i for i in (0, 1) if at[i] < n]
        ctx = make_ctx(cache, [slots[i] for i in live], [at[i] for i in live], [1] * len(live), F32, ws)
        out = torch.zeros(len(live), width, device=DEV)
        part.forward(d(torch.stack([(a, b)[i][at[i]] for i in live])), out, ctx, cache.layer(0), True)
        for r, i in enumerate(live):
            got[i][at[i]] = out[r]
            at[i] += 1
            cache.commit(slots[i], at[i])
    assert rel_err(got[0], wa) < 1e-4 and rel_err(got[1], wb) < 1e-4


def _blind_channel(W, p):
    """Channel 0 of the input reaches the values only, and only the current token's tap of their convolution: a large number
    there makes one position's value dwarf the others while its score stays ordinary, so whoever sees it shows it."""
    for name in ("q", "k"):
        W[p + name][:, 0] = 0.0
    W[p + "v.conv"][:, :-1] = 0.0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,kv,dim,vdim,size,conv", [(4, 2, 16, 24, 20, 3), (2, 2, 8, 8, 150, 4), (1, 1, 24, 24, 1, 1), (3, 1, 9, 17, 33, 2),
                                                         (4, 2, 64, 64, 70, 5), (2, 1, 128, 128, 129, 2), (6, 2, 64, 32, 64, 4)])
def test_window_edges_with_a_value_that_dwarfs_the_rest(dtype, heads, kv, dim, vdim, size, conv):
    """One position's value is made huge: the results differ by orders of magnitude between the last query that sees it and the
    first that does not.  The position lies on both sides of a page border.  As one prompt, with the later tokens one by
    one, and in portions whose borders fall inside the window and inside the filters."""
    width, n, cut = 128, 330, 150
    m = gm.left(heads=heads, kv=kv, dim=dim, vdim=vdim, scale=0.6 / math.sqrt(dim), conv=conv, size=size)
    part, W, p = _part("left", m, dtype, width, seed=dim + size, hot=1.5, edit=_blind_channel)
    cache, ws = _cache(part, dtype), _workspace()
    tol = 3e-5 if dtype == F32 else 3e-2
    for big in (63, 64, 130):
        x = (torch.randn(n, width, generator=torch.Generator().manual_seed(big)) * 0.3).to(dtype)
        x[big, 0] = 3e4
        want = pg.window_attention(x.double(), W, p, m)
        lost = big + size                                         # the first query that no longer sees `big`
        assert float(want[lost - 1].abs().max()) > 20 * float(want[lost].abs().max())
        assert rel_err(_drive(part, cache, x, [n], dtype, ws), want) < tol, big
        assert rel_err(_drive(part, cache, x, [cut, 1], dtype, ws), want) < tol, big
    assert rel_err(_drive(part, cache, x, [2, 1, 61, 3, 64, 7], dtype, ws), want) < tol
    for first in (1, 2, 5):                                       # the first tokens of a sequence alone
        assert rel_err(_drive(part, cache, x[:first], [1], dtype, ws), want[:first]) < tol


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,kv,dim,vdim,size", [(4, 2, 64, 64, 70), (2, 1, 128, 128, None), (3, 3, 24, 16, None), (16, 1, 64, 64, 200)])
def test_sink_takes_what_the_keys_leave(dtype, heads, kv, dim, vdim, size):
    """Queries and keys along one direction, so that all scores of a token are far below 0, near 0 or far above it: the
    sink takes everything, a share that depends on the number of keys, or nothing.  Leaving it out, or counting it per run of
    pages, changes the result by orders of magnitude.  Whole prompts, portions and single tokens (in 1 and in several runs)."""
    width, n = 96, 200

    def edit(W, p):
        for name in ("q", "k"):
            W[p + name].zero_()
            W[p + name][:, 0] = 1.0
            W[p + name + ".b"].zero_()
            W[p + name + ".conv"].zero_()
            W[p + name + ".conv"][:, -1] = 1.0
        W[p + "k"][:, 0] = 0.0
        W[p + "k"][:, 1] = 1.0
        W[p + "o.b"].zero_()
    m = gm.left(heads=heads, kv=kv, dim=dim, vdim=vdim, scale=1.0 / dim, conv=2, size=size)
    part, W, p = _part("left", m, dtype, width, seed=dim, edit=edit)
    x = (torch.randn(n, width, generator=torch.Generator().manual_seed(4)) * 0.5).to(dtype)
    x[:, 1] = 1.0                                                 # every key is the same; a query's channel 0 is its score
    x[:, 0] = torch.tensor([-40.0, -8.0, -3.0, 0.0, 3.0, 40.0]).repeat(n)[:n].to(dtype)
    want = pg.window_attention(x.double(), W, p, m)
    peak = want.abs().amax(-1)
    assert float(peak[180]) < 1e-10 * float(peak[185])            # scores -40 and 40
    cache, ws = _cache(part, dtype), _workspace()
    rows = [t for t in range(n) if t % 6]                         # those of score -40 are compared by size
    for portions in ([n], [130, 1], [64, 2, 66, 5]):
        got = _drive(part, cache, x, portions, dtype, ws)
        assert rel_err(got[rows], want[rows]) < (5e-5 if dtype == F32 else 3e-2), portions
        assert float(got[::6].abs().max()) < 1e-9 * float(peak.max())


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_members_are_normed_and_averaged(dtype):
    """The two mixers side by side: half the sum of the results, each RMS-normed over the width with its own weight, the
    attention's output bias inside its norm; whole and in portions."""
    width, n = 80, 140
    m = {"left": gm.left(heads=4, kv=2, dim=16, vdim=8, scale=0.3, conv=3, size=30),
         "right": gm.right(heads=3, kv=1, dim=12, vdim=20, conv=2)}

    def edit(W, p):
        W[p + "left.o.b"] *= 10.0
    part, W, p = _part("parallel", m, dtype, width, seed=2, edit=edit)
    x = torch.randn(n, width, generator=torch.Generator().manual_seed(1)).to(dtype)
    want = pg.side_by_side(x.double(), W, p, m, 1e-5)
    cache, ws = _cache(part, dtype), _workspace()
    for portions in ([n], [70, 3, 1], [2]):
        assert rel_err(_drive(part, cache, x, portions, dtype, ws), want) < PART_TOL[dtype], portions


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("experts,top,ff,count,keep", [(6, 3, 24, 3, 2), (8, 2, 64, 8, 3), (12, 5, 40, 2, 1), (1, 1, 16, None, None),
                                                       (4, 4, 20, 4, 4)])
def test_experts_as_a_part(dtype, experts, top, ff, count, keep):
    """The mixture against the plain one for 1, 7, 300 and 1,100 tokens.  bfloat16 runs pin the choice, float32 runs route
    freely."""
    width = 128
    mlp = gm.moe(experts=experts, top=top, ff=ff, count=count, keep=keep)
    part, W, p = _part("mlp", mlp, dtype, width, seed=experts + top, pin=dtype == BF16)
    ws = _workspace()
    for n in (1, 7, 300, 1100):
        x = torch.randn(n, width, generator=torch.Generator().manual_seed(n))
        if dtype == BF16:
            x[:, 0] = 2.0
        x = x.to(dtype)
        got = torch.zeros(n, width, device=DEV)
        part.forward(d(x), got, _Scratch(ws, dtype))
        assert rel_err(got, pg.experts_ff(x.double(), W, p, mlp)) < (3e-5 if dtype == F32 else 2e-2), n


# ---------------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    made = {}

    def get(name, dtype="bfloat16", seed=0):
        pin = dtype == "bfloat16"                 # float32 runs route freely
        if (name, pin, seed) not in made:
            made[(name, pin, seed)] = gm.make(tmp_path_factory.mktemp("gatarax"), name, seed=seed, pin=pin)
        return made[(name, pin, seed)]
    return get


def _engine(model, dtype, **kw):
    from rust_inference_b200.engine.engine import Engine
    return Engine.from_pretrained(model.folder, dtype=dtype, max_tokens=kw.pop("max_tokens", 2048), n_slots=kw.pop("n_slots", 6), **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_whole_prompt_layers_and_decoding(dtype, name, models):
    """A whole prompt (the stream after every layer too), the same with its last tokens one by one (across the edges of
    windows and pages), and a slot used again: its states must start at zero, its pages hold old rows."""
    model = models(name, dtype)
    eng = _engine(model, dtype)
    tokens = random_tokens(230, model.cfg["vocab"], 1)
    streams = []
    want = model.plain_logits(tokens, streams=streams)
    tol = TOL[dtype]
    probe = Streams()
    s = eng.alloc_slot()
    got = eng.step([s], [tokens], "all", probe=probe)
    assert rel_err(got, want) < tol
    assert len(probe.seen) == len(streams) == len(model.cfg["layers"])
    for a, b in zip(probe.seen, streams):
        assert rel_err(a, b) < tol
    eng.free_slot(s)
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
        assert rel_err(_run(eng, s, tokens, portions), want) < TOL[dtype], portions
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
        assert rel_err(torch.cat(got[b]), want[b]) < TOL[dtype], b
    assert second is not None and second < TOL[dtype]
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


def test_a_batch_that_decodes_beyond_the_low_rank_kernel_s_tokens(models):
    """Twenty sequences decode together: more tokens than the preparing kernel forms low-rank maps for, so a captured step takes
    them as products."""
    model = models("A", "float32")
    eng = _engine(model, "float32", n_slots=24, max_tokens=24 * 64)
    seqs = [random_tokens(4 + i % 5 + 9, model.cfg["vocab"], 200 + i) for i in range(20)]
    slots = [eng.alloc_slot() for _ in seqs]
    eng.step(slots, [t[:-9] for t in seqs], "none")
    rows = [[] for _ in seqs]
    for k in range(9):
        out = eng.step(slots, [[t[len(t) - 9 + k]] for t in seqs], "last").cpu()
        for b in range(20):
            rows[b].append(out[b:b + 1])
    assert eng.decode_graph(20).graph is not None
    for b, t in enumerate(seqs):
        assert rel_err(torch.cat(rows[b]), model.plain_logits(t)[-9:]) < TOL["float32"], b


def test_what_carries_a_far_token(tmp_path):
    """The first token lies outside every window of a late position: with states that forget at once the late logits do not
    depend on it (the convolutions reach back a few tokens per layer only); with a slow delta rule, a slow fixed decay or
    an attention without a window they do.  The engine agrees with the plain model in every case."""
    def par(size):
        return gm.parallel(gm.left(heads=2, kv=1, dim=16, vdim=16, scale=0.25, conv=3, size=size),
                           gm.right(heads=2, kv=1, dim=16, vdim=8, conv=2), gm.dense(40))

    def light(c):
        return gm.lightning(heads=2, dim=16, vdim=16, decay=(c, c), mlp=gm.dense(40))

    def forget(fast):
        def edit(W):
            for k in W:
                if k.endswith("right.A_log"):
                    W[k].fill_(4.0 if fast else -8.0)
                if k.endswith("right.dt_bias"):
                    W[k].fill_(4.0 if fast else -1.0)
                if k.endswith("right.a2"):
                    W[k].mul_(0.1)
        return edit
    cases = (("windows", [par(9), par(9), light(0.0)], True, False), ("delta", [par(9), par(9)], False, True),
             ("decay", [par(9), light(0.9999)], True, True), ("no_window", [par(None), par(9)], True, True))
    for name, layers, fast, reaches in cases:
        cfg = gm.model(vocab=97, width=64, eps=1e-6, taps=3, scale=1.0, logit_scale=1.0, layers=layers)
        model = gm.make(tmp_path, name, cfg=cfg, edit=forget(fast))
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
        assert list(g.tokens) == pg.greedy(model.cfg, model.weights, p, n_new)
    lefts = [L["mixer"]["left"] for L in model.cfg["layers"] if L["type"] == "parallel"]
    assert m.memory()["cache_bytes_per_position"] == sum(a["kv_heads"] * (a["dim"] + a["vdim"]) * 4 for a in lefts)


@pytest.mark.parametrize("name", ["A", "B"])
def test_state_dict_round_trip(name, models):
    """The tensors come back apart under the file's names."""
    from rust_inference_b200 import Model
    model = models(name)
    m = Model.load(model.folder, dtype="float32", max_tokens_in_cache=512)
    sd = m.state_dict()
    assert set(sd) == set(model.weights)
    for k, v in model.weights.items():
        assert torch.equal(sd[k].float().cpu().reshape(v.shape), v), k


def test_trace_replay_picks_the_model_by_its_config(models, tmp_path):
    """`bin/trace_run` on a Gatarax folder: two requests start together, go on by one token and end at different steps; then
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


def test_the_command_line_on_a_gatarax_folder(models):
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
    assert [[int(t) for t in l.split()] for l in lines] == [pg.greedy(model.cfg, model.weights, q, 6) for q in prompts]


@pytest.mark.parametrize("dim", [64, 128])
def test_tensor_core_kernels_take_the_sink(dim, monkeypatch):
    """bfloat16 heads of 64 and 128 channels with a sink: prompts on the tcgen05 kernel, single tokens on the decode kernel with
    the forms of the score (one run of pages and several); neither the generic nor the mma.sync prompt kernel is called."""
    from rust_inference_b200.kernels import ops

    def refuse(*a, **k):
        raise AssertionError("another attention kernel was called")
    width, n = 128, 420
    m = gm.left(heads=4, kv=2, dim=dim, vdim=dim, scale=0.8 / math.sqrt(dim), conv=3, size=300)
    part, W, p = _part("left", m, BF16, width, seed=dim, hot=1.5)
    x = (torch.randn(n, width, generator=torch.Generator().manual_seed(3)) * 0.3).to(BF16)
    want = pg.window_attention(x.double(), W, p, m)
    cache, ws = _cache(part, BF16), _workspace()
    monkeypatch.setattr(ops, "attention_generic", refuse)
    monkeypatch.setattr(ops, "attention_prefill_forms", refuse)
    for splits in ("1", "3", None):
        if splits is None:
            monkeypatch.delenv("RI_B200_DECODE_SPLITS")
        else:
            monkeypatch.setenv("RI_B200_DECODE_SPLITS", splits)
        assert rel_err(_drive(part, cache, x, [380, 1], BF16, ws), want) < 3e-2
