"""Pagulix without a GPU: the configuration reader and its errors, the tensors the model declares against the plain list,
cache requests, rotation tables, and the plain restatement's mechanisms against closed forms."""
import copy
import math

import numpy as np
import pytest
import torch

import pagulix_models as gm
import plain_pagulix as pp
from rust_inference_b200.cache.sequence_cache import KVRequest, SequenceCache, StateRequest
from rust_inference_b200.config.model_config import ConfigError
from rust_inference_b200.config.registry import config_from_dict, get_architecture, load_spec, registered_architectures
from rust_inference_b200.engine.model import DecoderModel, declared_tensors
from rust_inference_b200.parts.rope import rope_tables, stretched_frequencies


def _spec(cfg):
    return get_architecture("Pagulix").build_spec(config_from_dict(cfg))


def test_registered_and_round_trip():
    assert "Pagulix" in registered_architectures()
    for cfg in gm.CONFIGS.values():
        parsed = config_from_dict(cfg)
        again = config_from_dict(parsed.to_dict())
        assert again.to_dict() == parsed.to_dict()
        assert [(L.mixer, L.mlp) for L in again.layers] == [(L.mixer, L.mlp) for L in parsed.layers]


@pytest.mark.parametrize("name", list(gm.CONFIGS))
def test_declared_tensors_equal_the_plain_list(name, tmp_path):
    """But for the blending number of the first blending layer, which nothing reads."""
    cfg = gm.CONFIGS[name]
    _, spec = load_spec(gm.make(tmp_path, name).folder)
    declared = {k: tuple(v.shape) for k, v in declared_tensors(spec).items()}
    plain = pp.tensor_shapes(cfg)
    unread = {k for k in plain if k not in declared}
    mixing = [i for i, L in enumerate(cfg["layers"]) if L["mixer"].get("v_mix")]
    assert unread == ({f"l{mixing[0]}.mix.vmix"} if mixing else set()) and unread <= set(spec.ignored_tensors)
    assert declared == {k: v for k, v in plain.items() if k not in unread}
    assert spec.streams == cfg["streams"]


def test_cache_requests():
    """A latent layer asks for one row per position in a group of its window, attention for keys and values, the delta rule for
    its state and its convolutions' inputs, which start at zero in a slot used again."""
    model = DecoderModel(_spec(gm.CONFIGS["A"]), dtype=torch.float32, device="cpu")
    reqs = model.cache_requests()
    assert reqs[0] == KVRequest(2, 16, None, 24) and reqs[3] == KVRequest(2, 24, None, None)
    assert reqs[1] == (StateRequest((4, 16, 24)), StateRequest((2, 2 * 2 * 16 + 4 * 24)))
    assert reqs[2] == KVRequest(1, 48, 20, 40, True)
    cache = SequenceCache(reqs, max_tokens=256, max_seq_len=128, dtype=torch.float32, device="cpu", n_slots=2)
    state, conv = cache.layer(1).parts
    slot = cache.alloc_slot()
    state.state[slot].fill_(3.0)
    conv.state[slot].fill_(3.0)
    cache.free_slot(slot)
    assert cache.alloc_slot() == slot
    assert float(state.state[slot].abs().sum()) == 0.0 and float(conv.state[slot].abs().sum()) == 0.0


def test_tensors_of_an_absent_feed_forward_may_be_in_the_file():
    import fnmatch
    ignored = _spec(gm.CONFIGS["A"]).ignored_tensors
    for name in ("l1.norm2", "l1.ls2", "l1.hc2.mix"):
        assert any(fnmatch.fnmatchcase(name, p) for p in ignored)
    assert not any(fnmatch.fnmatchcase("l0.norm2", p) for p in ignored)


@pytest.mark.parametrize("edit,message", [
    (lambda c: c.pop("streams"), "lacks 'streams'"),
    (lambda c: c.update(streams=0), "streams must be an integer >= 1"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c.update(logit_softcap=0.0), "logit_softcap must be positive"),
    (lambda c: c["norm"].update(eps=-1.0), "eps"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), r"layers\[0\]\.mixer lacks 'scale'"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"].update(v_mix="yes"), "v_mix must be true or false"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=16), "cannot be blended with those of layer 0"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "even and at most 16"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("original"), r"scaling lacks 'original'"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(high=1.0), "high must be above low"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=6), "must be the size of the rotated part, 8"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][2]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), r"layers\[1\]\.mixer lacks 'conv'"),
    (lambda c: c["layers"][1].update(type="lightning"), "not a mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "not a feed-forward"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "cannot give 7 choices"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "shared lacks 'ff'"),
])
def test_configuration_errors_name_the_key(edit, message):
    cfg = copy.deepcopy(gm.CONFIGS["A"])
    edit(cfg)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(cfg)


def test_streams_and_parts_that_do_not_go_together():
    from rust_inference_b200.parts.registry import lookup
    kw = dict(hidden_size=8, dtype=torch.float32, device="cpu")
    with pytest.raises(ValueError, match="between 1 and"):
        lookup("stream_link", "stream_link")(streams=0, **kw)
    link, other = (lookup("stream_link", "stream_link")(streams=s, **kw) for s in (2, 3))
    arrangement = lookup("arrangement", "parallel_streams")
    with pytest.raises(ValueError, match="comes with its norm and link"):
        arrangement(mixer=object(), mixer_norm=object(), mixer_link=link, feed_forward=object())
    with pytest.raises(ValueError, match="same streams"):
        arrangement(mixer=object(), mixer_norm=object(), mixer_link=link, feed_forward=object(), feed_forward_norm=object(),
                    feed_forward_link=other)
    with pytest.raises(ValueError, match="'first' or 'mixed'"):
        lookup("mixer", "gqa_attention")(n_heads=1, n_kv_heads=1, head_dim=8, qkv_bias=False, value_mix="second",
                                         position=gm_position(8), **kw)


def gm_position(dim):
    from rust_inference_b200.parts.spec import PartSpec
    return PartSpec("rope", {"head_dim": dim, "base": 100.0})


# ---- rotation ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dims,base,factor,low,high,original", [(48, 5e5, 16.0, 1.0, 5.0, 4096.0), (16, 500.0, 4.0, 1.0, 3.0, 100.0),
                                                               (24, 10000.0, 32.0, 0.5, 9.0, 64.0), (2, 10.0, 2.0, 1.0, 2.0, 1.0)])
def test_stretched_waves(dims, base, factor, low, high, original):
    """Kept, blended and slowed channels against the plain form, and the tables of cos and sin that are made from them."""
    scaling = dict(factor=factor, low=low, high=high, original=original)
    got = stretched_frequencies(dims, base, **scaling)
    want = pp.stretched(pp.frequencies(dims, base), scaling).numpy()
    assert np.allclose(got, want, rtol=1e-12)
    cos, sin = rope_tables(dims, base, 300, True, wave_scaling=scaling)
    assert cos.dtype == np.float32 and np.abs(cos - np.cos(np.arange(300)[:, None] * want)).max() < 1e-7
    assert np.abs(sin - np.sin(np.arange(300)[:, None] * want)).max() < 1e-7


def test_stretched_waves_have_all_three_kinds():
    f = pp.frequencies(48, 5e5)
    s = dict(factor=16.0, low=1.0, high=5.0, original=4096.0)
    ratio = (f / pp.stretched(f, s)).tolist()
    assert ratio[0] == 1.0 and abs(ratio[-1] - 16.0) < 1e-9
    assert any(1.001 < r < 15.999 for r in ratio)


def test_norm_without_weights_commutes_with_a_rotation():
    x = _r(5, 2, 12)
    f = pp.frequencies(8, 50.0)
    for interleaved in (False, True):
        assert torch.allclose(pp.unit_rms(pp.rotate(x, f, interleaved), 1e-5), pp.rotate(pp.unit_rms(x, 1e-5), f, interleaved))


# ---- the plain mechanisms against closed forms ---------------------------------------------------------------
def _r(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def test_plain_rotation_pairs():
    x = _r(3, 1, 6)
    f = torch.tensor([0.5, 0.1], dtype=torch.float64)
    a = 2 * f
    y = pp.rotate(x, f, interleaved=True)[2, 0]
    assert abs(float(y[2]) - float(x[2, 0, 2] * math.cos(a[1]) - x[2, 0, 3] * math.sin(a[1]))) < 1e-12
    y = pp.rotate(x, f, interleaved=False)[2, 0]
    assert abs(float(y[3]) - float(x[2, 0, 3] * math.cos(a[1]) + x[2, 0, 1] * math.sin(a[1]))) < 1e-12
    assert torch.equal(y[4:], x[2, 0, 4:])


def test_plain_sink():
    s = torch.tensor([[[1.3]]], dtype=torch.float64)
    ok = torch.ones(1, 1, dtype=torch.bool)
    w = pp.masked_softmax(s, ok, torch.tensor([0.4], dtype=torch.float64))
    assert abs(float(w) - math.exp(1.3) / (math.exp(1.3) + math.exp(0.4))) < 1e-12
    assert float(pp.masked_softmax(s, ok)) == 1.0
    assert float(pp.masked_softmax(s, ok, torch.tensor([800.0], dtype=torch.float64))) == 0.0


def test_plain_latent_attention_equals_the_absorbed_form():
    """Scores of queries carried into the latent space, and the heads' maps applied to the mixed latents."""
    m = gm.latent(heads=2, dim=3, rot_dim=4, vdim=5, rank=6, scale=0.4, size=3)
    cfg = gm.model(vocab=7, width=8, streams=1, factor=1.0, cap=1.0, eps=1e-5, layers=[gm.layer("latent", m)])
    W = {k: v.double() for k, v in pp.random_weights(cfg, 1).items()}
    p, h = "l0.mix.", _r(5, 8)
    f = pp.frequencies(4, 10000.0)
    q = (h @ W[p + "q"].T).view(5, 2, 7)
    down = h @ W[p + "dkv"].T
    c = pp.rms_norm(down[:, :6], W[p + "dkv.norm"], 1e-5)
    kr = pp.rotate(down[:, None, 6:], f, True)[:, 0]
    out = torch.zeros(5, 2, 5, dtype=torch.float64)
    for t in range(5):
        for hd in range(2):
            uk, uv = W[p + "uk"][3 * hd:3 * hd + 3], W[p + "uv"][5 * hd:5 * hd + 5]
            wide = torch.cat([uk.T @ q[t, hd, :3], pp.rotate(q[:, hd:hd + 1, 3:], f, True)[t, 0]])
            e = {s: math.exp(0.4 * float(wide @ torch.cat([c[s], kr[s]]))) for s in range(max(0, t - 2), t + 1)}
            total = sum(e.values()) + math.exp(float(W[p + "sink"][hd]))
            out[t, hd] = uv @ sum(e[s] / total * c[s] for s in e)
    assert torch.allclose(pp.latent_attention(h, W, p, m, 1e-5), out.reshape(5, 10) @ W[p + "o"].T, atol=1e-12)


def test_plain_values_are_blended_with_the_first_layer_s():
    m = gm.attention(heads=2, kv=1, dim=4, vdim=3, scale=0.5, dims=4, mix=True)
    cfg = gm.model(vocab=7, width=6, streams=1, factor=1.0, cap=1.0, eps=1e-5, layers=[gm.layer("attention", m), gm.layer("attention", m)])
    W = {k: v.double() for k, v in pp.random_weights(cfg, 1).items()}
    h, shared = _r(1, 6), {}
    pp.attention(h, W, "l0.mix.", m, 1e-5, shared)
    lam = float(W["l1.mix.vmix"])
    v = (1 - lam) * (W["l1.mix.v"] @ h[0]) + lam * (W["l0.mix.v"] @ h[0])     # one token: attention hands its value through
    assert torch.allclose(pp.attention(h, W, "l1.mix.", m, 1e-5, shared)[0], W["l1.mix.o"] @ torch.cat([v, v]), atol=1e-12)


def test_plain_delta_rule_replaces_a_value():
    """With no decay and step 1, writing a second value under the same unit key leaves only the second."""
    d, dv, D = 3, 2, 4
    W = {k: torch.zeros(s, dtype=torch.float64) for k, s in {
        "q": (d, D), "k": (d, D), "v": (dv, D), "b": (1, D), "a": (1, D), "g": (dv, D)}.items()}
    W["q"][0, 0] = W["k"][0, 0] = 50.0
    W["v"][:, 1:3] = torch.eye(2, dtype=torch.float64) * 5
    W["b"][0, 0] = 100.0
    W["g"][:, 0] = 1.0
    W["o"] = torch.eye(dv, dtype=torch.float64)
    W.update({n + ".conv": torch.ones(r, 1, dtype=torch.float64) for n, r in (("q", d), ("k", d), ("v", dv))})
    W.update({"A_log": torch.full((1,), -60.0, dtype=torch.float64), "dt_bias": torch.zeros(1, dtype=torch.float64),
              "norm": torch.ones(dv, dtype=torch.float64)})
    h = torch.tensor([[1.0, 1.0, 0.0, 0.0], [1.0, 0.0, 1.0, 0.0]], dtype=torch.float64)
    y = pp.delta_rule(h, W, "", {"heads": 1, "kv_heads": 1, "dim": d, "vdim": dv}, 1e-12)
    gate = 1.0 / (1.0 + math.exp(-1.0))
    assert torch.allclose(y, gate * math.sqrt(2.0) * torch.eye(2, dtype=torch.float64), atol=1e-6)


def test_plain_router():
    """The bias decides the choice and enters the weights, which only the chosen logits share."""
    ids, w = pp.route(torch.ones(1, 1, dtype=torch.float64), torch.tensor([[1.0], [2.0], [0.0]], dtype=torch.float64),
                      torch.tensor([0.0, -5.0, 0.5], dtype=torch.float64), 2)
    assert ids[0].tolist() == [0, 2]
    assert torch.allclose(w[0], torch.softmax(torch.tensor([1.0, 0.5], dtype=torch.float64), 0))


def test_plain_streams_are_written_from_the_old_ones():
    x, y = _r(2, 1, 3), _r(1, 3, seed=1)
    mix = torch.tensor([[0.0, 2.0], [1.0, 0.0]], dtype=torch.float64)        # [from, to]: exchanged, one of them doubled
    out = torch.tensor([1.0, 0.5], dtype=torch.float64)
    new = pp.write_streams(x, mix, out, y, 0.1)
    assert torch.allclose(new[0], x[1] + 0.1 * y) and torch.allclose(new[1], 2.0 * x[0] + 0.05 * y)
    assert torch.allclose(pp.read_streams(x, torch.tensor([2.0, -1.0], dtype=torch.float64)), 2.0 * x[0] - x[1])
