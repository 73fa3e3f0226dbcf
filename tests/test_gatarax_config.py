"""Gatarax without a GPU: the configuration reader and its errors, the tensors the model declares against the plain list,
cache requests, ranks that tensors' shapes give, and the plain restatement's mechanisms against closed forms."""
import copy
import math

import pytest
import torch

import gatarax_models as gm
import plain_gatarax as pg
from rust_inference_b200.cache.sequence_cache import KVRequest, SequenceCache, StateRequest
from rust_inference_b200.config.model_config import ConfigError
from rust_inference_b200.config.registry import config_from_dict, get_architecture, load_spec, registered_architectures
from rust_inference_b200.engine.model import DecoderModel, declared_tensors


def _spec(cfg):
    arch = get_architecture("Gatarax")
    return arch.build_spec(arch.parse_config(cfg, shapes=pg.tensor_shapes(cfg)))


def test_registered_and_round_trip():
    assert "Gatarax" in registered_architectures()
    for cfg in gm.CONFIGS.values():
        parsed = get_architecture("Gatarax").parse_config(cfg, shapes=pg.tensor_shapes(cfg))
        again = config_from_dict(parsed.to_dict())              # the ranks are written out: no shapes needed
        assert again.to_dict() == parsed.to_dict()
        assert [(L.mixer, L.mlp) for L in again.layers] == [(L.mixer, L.mlp) for L in parsed.layers]


@pytest.mark.parametrize("name", list(gm.CONFIGS))
def test_declared_tensors_equal_the_plain_list(name):
    cfg = gm.CONFIGS[name]
    assert {k: tuple(v.shape) for k, v in declared_tensors(_spec(cfg)).items()} == pg.tensor_shapes(cfg)


def test_cache_requests():
    """A layer asks for its mixer's needs and, beside them, for the inputs its two convolutions share; of a parallel mixer the
    attention asks for keys, values and its projections' last rows, the delta rule for its state and convolutions."""
    model = DecoderModel(_spec(gm.CONFIGS["A"]), dtype=torch.float32, device="cpu")
    reqs = model.cache_requests()
    assert reqs[0] == (((KVRequest(2, 16, 20, 24), StateRequest((2, 4 * 16 + 2 * 16 + 2 * 24))),
                        (StateRequest((4, 16, 24)), StateRequest((1, 2 * 2 * 16 + 4 * 24)))), StateRequest((3, 96)))
    assert reqs[1] == (StateRequest((3, 16, 8)), StateRequest((3, 96)))
    cache = SequenceCache(reqs, max_tokens=256, max_seq_len=128, dtype=torch.float32, device="cpu", n_slots=2)
    (keys, proj), (state, conv) = (part.parts for part in cache.layer(0).parts[0].parts)
    assert tuple(keys.k.shape[1:]) == (2, 64, 16) and tuple(keys.v.shape[1:]) == (2, 64, 24)
    slot = cache.alloc_slot()
    shared = cache.layer(0).parts[1]
    for layer in (proj, state, conv, shared):
        layer.state[slot].fill_(3.0)
    cache.free_slot(slot)
    assert cache.alloc_slot() == slot
    assert all(float(layer.state[slot].abs().sum()) == 0.0 for layer in (proj, state, conv, shared))
    # one tap carries nothing
    assert DecoderModel(_spec(gm.CONFIGS["B"]), dtype=torch.float32, device="cpu").cache_requests()[0][1] == StateRequest((0, 72))


def test_ranks_from_shapes(tmp_path):
    cfg = gm.CONFIGS["A"]
    with pytest.raises(ConfigError, match=r"layers\[0\]\.mixer\.right\.decay_rank"):
        config_from_dict(cfg)
    made = gm.make(tmp_path, "A", ranks=lambda i: (7, 1))
    _, spec = load_spec(made.folder)
    assert {k: tuple(v.shape) for k, v in declared_tensors(spec).items()} == pg.tensor_shapes(cfg, lambda i: (7, 1))


def test_a_convolution_nobody_reads_behind_may_be_in_the_file():
    assert "l1.canon2" in _spec(gm.CONFIGS["A"]).ignored_tensors and "l0.canon2" not in _spec(gm.CONFIGS["A"]).ignored_tensors


@pytest.mark.parametrize("edit,message", [
    (lambda c: c.pop("canon"), "canon"),
    (lambda c: c["canon"].update(taps=0), "canon.taps"),
    (lambda c: c.pop("logit_scale"), "logit_scale"),
    (lambda c: c["embedding"].pop("scale"), "embedding lacks 'scale'"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), r"layers\[0\]\.mixer\.left lacks 'scale'"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(kv_heads=3), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("conv"), r"right lacks 'conv'"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "lacks 'right'"),
    (lambda c: c["layers"][0].update(type="attention"), "not a mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "not a feed-forward"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "cannot give 5 choices"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "equal groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].pop("keep"), "keep"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.5]), "one number for each of the 3 heads"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, "x", 1]), "must be numbers"),
])
def test_configuration_errors_name_the_key(edit, message):
    cfg = copy.deepcopy(gm.CONFIGS["A"])
    edit(cfg)
    with pytest.raises(ConfigError, match=message):
        get_architecture("Gatarax").parse_config(cfg, shapes=pg.tensor_shapes(gm.CONFIGS["A"]))


# ---- the plain mechanisms against closed forms ---------------------------------------------------------------
def _r(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def test_plain_convolution():
    x, w = _r(6, 2), _r(2, 3, seed=1)
    y = pg.short_conv(x, w)
    for t in range(6):
        for c in range(2):
            want = sum(float(w[c, j]) * float(x[t - 2 + j, c]) for j in range(3) if t - 2 + j >= 0)
            assert abs(float(y[t, c]) - want) < 1e-12
    assert torch.allclose(pg.short_conv(x[:1], w), x[:1] * w[:, 2])          # shorter than the filter
    assert torch.allclose(pg.input_conv(x, torch.zeros(2, 3, dtype=torch.float64)), x)


def test_plain_sink_and_window():
    """One visible key of score s gets e^s / (1 + e^s); two equal ones of score 0 a third each."""
    s = torch.tensor([[[1.3]]], dtype=torch.float64)
    ok = torch.ones(1, 1, dtype=torch.bool)
    assert abs(float(pg.sink_weights(s, ok)) - 1 / (1 + math.exp(-1.3))) < 1e-12
    assert torch.allclose(pg.sink_weights(torch.zeros(1, 2, 2, dtype=torch.float64), torch.ones(2, 2, dtype=torch.bool)),
                          torch.full((1, 2, 2), 1 / 3, dtype=torch.float64))
    assert float(pg.sink_weights(torch.tensor([[[-800.0]]], dtype=torch.float64), ok)) == 0.0
    assert float(pg.sink_weights(torch.tensor([[[800.0]]], dtype=torch.float64), ok)) == 1.0


def test_plain_delta_rule_replaces_a_value():
    """With no decay and step 1, writing a second value under the same unit key leaves only the second."""
    d, dv, D = 3, 2, 4
    W = {k: torch.zeros(s, dtype=torch.float64) for k, s in {
        "q": (d, D), "k": (d, D), "v": (dv, D), "b": (1, D), "a1": (1, D), "a2": (d, 1), "g1": (1, D), "g2": (dv, 1), "o": (dv, dv)}.items()}
    W["q"][0, 0] = W["k"][0, 0] = 50.0
    W["v"][:, 1:3] = torch.eye(2, dtype=torch.float64) * 5
    W["b"][0, 0] = 100.0
    W["o"] = torch.eye(dv, dtype=torch.float64)
    W.update({n + ".conv": torch.ones(r, 1, dtype=torch.float64) for n, r in (("q", d), ("k", d), ("v", dv))})
    W.update({"A_log": torch.full((1,), -60.0, dtype=torch.float64), "dt_bias": torch.zeros(d, dtype=torch.float64),
              "norm": torch.ones(dv, dtype=torch.float64)})
    h = torch.tensor([[1.0, 1.0, 0.0, 0.0], [1.0, 0.0, 1.0, 0.0]], dtype=torch.float64)
    y = pg.delta_rule(h, W, "", {"heads": 1, "kv_heads": 1, "dim": d, "vdim": dv}, 1e-12)
    assert torch.allclose(y, 0.5 * math.sqrt(2.0) * torch.eye(2, dtype=torch.float64), atol=1e-6)     # unit rms, gate 1/2


def test_plain_decays_act_on_key_channels():
    W = {"a1": _r(2, 3), "a2": _r(8, 2, seed=1), "dt_bias": _r(8, seed=2), "A_log": _r(2, seed=3)}
    h = _r(5, 3, seed=4)
    g = pg.channel_decays(h, W, "", 2, 4)
    z = W["a2"][6] @ (W["a1"] @ h[3]) + W["dt_bias"][6]              # head 1, channel 2
    assert abs(float(g[3, 1, 2]) - math.exp(-math.exp(float(W["A_log"][1])) * math.log1p(math.exp(float(z))))) < 1e-12


def test_plain_lightning_sums_decayed_products():
    m = {"heads": 2, "dim": 3, "vdim": 2, "decay": [0.5, 1.0]}
    W = {"q": _r(6, 4), "k": _r(6, 4, seed=1), "v": _r(4, 4, seed=2), "g": torch.zeros(4, 4, dtype=torch.float64),
         "norm": torch.ones(4, dtype=torch.float64), "o": torch.eye(4, dtype=torch.float64)}
    h = _r(5, 4, seed=3)
    q, k, v = (pg.silu(h @ W[n].T).view(5, 2, -1) for n in ("q", "k", "v"))
    o = torch.zeros(5, 2, 2, dtype=torch.float64)
    for t in range(5):
        for s in range(t + 1):
            for head in range(2):
                o[t, head] += m["decay"][head] ** (t - s) * (q[t, head] @ k[s, head]) * v[s, head]
    want = 0.5 * pg.unit_rms(o.reshape(5, 4), 1e-6)                  # gate sigmoid(0)
    assert torch.allclose(pg.lightning(h, W, "", m, 1e-6), want, atol=1e-9)


def test_plain_router_ranks_groups_by_their_best_score():
    """Two good experts in one group lose against the single best ones of two others."""
    logits = torch.tensor([[2.0, 1.9, 2.1, -5.0, 2.2, -5.0]], dtype=torch.float64)
    ids, w = pg.route(torch.ones(1, 1, dtype=torch.float64), logits.T, top=2, groups=3, keep=2)
    assert sorted(ids[0].tolist()) == [2, 4]
    s = torch.softmax(logits, -1)[0]
    assert torch.allclose(w[0], s[ids[0]])                          # the scores over all experts, as they are


def test_plain_dense_activation():
    W = {"up": torch.eye(2, dtype=torch.float64), "down": torch.eye(2, dtype=torch.float64)}
    assert torch.equal(pg.dense_ff(torch.tensor([[-3.0, 2.0]], dtype=torch.float64), W, ""), torch.tensor([[0.0, 4.0]], dtype=torch.float64))
