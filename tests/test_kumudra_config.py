"""The Kumudra configuration without a GPU: config.json keys to layers as data, tensor names, loops
with a state per pass, what the configuration refuses, and the plain implementation's own properties."""

import copy
import math

import pytest
import torch

import kumudra_util as U
from plain import kumudra_plain as P


def build(cfg):
    from scratch_llm_b200.config import config_from_dict
    from scratch_llm_b200.engine.model import build_model
    return build_model(config_from_dict(cfg))


@pytest.mark.parametrize("name", list(U.CONFIGS))
def test_tensor_names_are_those_of_the_random_model(name):
    cfg = U.CONFIGS[name]
    specs = build(cfg).param_specs()
    tensors = U.random_tensors(cfg, 0)
    assert set(specs) == set(tensors)
    for key, spec in specs.items():
        got = tuple(tensors[key].shape)
        assert len(got) == len(spec.shape)
        assert all(w in (-1, g) for g, w in zip(got, spec.shape)), key


def test_looped_layers_have_a_cache_entry_and_a_state_per_pass():
    model = build(U.CONFIGS["S"])
    assert [(r.layer, r.cache, r.write) for r in model.spec.order] == \
        [(0, 0, True), (1, 1, True), (2, 2, True), (1, 3, True), (2, 4, True)]
    assert [r.layer for r in model.spec.order] == P.run_order(U.CONFIGS["S"])
    kv, st = model.cache_specs()
    assert [k is not None for k in kv] == [False, True, False, True, False]
    # keys of 12 and values of 20 share pages of 32; the window is kept
    assert (kv[1].n_kv_heads, kv[1].head_dim, kv[1].window) == (2, 32, 13) and kv[1] == kv[3]
    assert tuple(st[0].shape) == (3, 6, 10) and tuple(st[2].shape) == (2, 11, 9)
    # time mixing: the matrix, and the previous token's input of the mixer
    assert [tuple(s.shape) for s in st[1]] == [(3, 14, 14), (48,)]
    for s in (st[0], st[1][0], st[1][1], st[2]):
        assert s.dtype == torch.float32
    assert model.spec.streams == 3 and model.spec.tie_embeddings


def test_every_loop_and_no_loop():
    for loop, want in ((None, [0, 1, 2]), ((0, 3, 1), [0, 1, 2]), ((1, 1, 4), [0, 1, 2]),
                       ((0, 1, 3), [0, 0, 0, 1, 2]), ((2, 3, 2), [0, 1, 2, 2]),
                       ((0, 3, 2), [0, 1, 2, 0, 1, 2])):
        cfg = U.config(50, 32, [U.gla(1, 4, 4), U.lightning(1, 4, 4, [0.5]), U.gla(2, 4, 4)],
                       loop=loop)
        model = build(cfg)
        assert [r.layer for r in model.spec.order] == want == P.run_order(cfg)
        assert [r.cache for r in model.spec.order] == list(range(len(want)))


def test_round_trip_and_refusals():
    from scratch_llm_b200.config import KumudraConfig, config_from_dict
    for name in U.CONFIGS:
        cfg = config_from_dict(U.CONFIGS[name])
        assert isinstance(cfg, KumudraConfig)
        again = config_from_dict(cfg.to_dict())
        assert again == cfg and again.model_spec() == cfg.model_spec()

    bad = [lambda c: c["layers"][0].update(type="attention"),
           lambda c: c["layers"][0]["mixer"].update(tau=0.0),
           lambda c: c["layers"][0]["mixer"].update(heads=0),
           lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3),
           lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=7),
           lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=14),
           lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("low"),
           lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].update(low=5.0),
           lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0),
           lambda c: c["layers"][1]["mixer"]["left"].pop("scale"),
           lambda c: c["layers"][1]["mixer"].pop("right"),
           lambda c: c["layers"][1]["mixer"].pop("left_scale"),
           lambda c: c["layers"][2]["mixer"].update(decay=[0.5]),
           lambda c: c["layers"][2]["mixer"].update(decay=[0.5, 1.5]),
           lambda c: c["layers"][0]["mlp"].update(kind="shared"),
           lambda c: c["layers"][0]["mlp"]["router"].update(top=7),
           lambda c: c["layers"][0]["mlp"]["router"].pop("scale"),
           lambda c: c["layers"][1]["mlp"].update(ff=0),
           lambda c: c["loop"].update(stop=4),
           lambda c: c["loop"].update(start=3, stop=2),
           lambda c: c["loop"].update(times=0),
           lambda c: c.update(streams=0),
           lambda c: c.pop("norm")]
    for change in bad:
        c = copy.deepcopy(U.CONFIGS["S"])
        change(c)
        with pytest.raises(ValueError):
            build(c)


def test_rotary_frequencies_scale_as_in_the_plain_model():
    from scratch_llm_b200.parts.position import Rotary
    sc = U.scaling(8.0, 1.0, 4.0, 200)
    rot = {"base": 700.0, "dims": 24, "scaling": sc}
    freqs = P.frequencies(rot)
    plain = P.frequencies({"base": 700.0, "dims": 24})
    kept = [f == g for f, g in zip(freqs, plain)]
    slowed = [abs(f * 8.0 - g) < 1e-15 for f, g in zip(freqs, plain)]
    assert any(kept) and any(slowed) and not all(k or s for k, s in zip(kept, slowed))
    table = Rotary(32, 700.0, 300, interleaved=False, rot_dims=24, llama3=sc)
    cos, sin = table.tables()
    assert cos.shape == (300, 12)
    for p in (0, 1, 17, 299):
        for i, f in enumerate(freqs):
            assert abs(float(cos[p, i]) - math.cos(p * f)) < 2e-5
            assert abs(float(sin[p, i]) - math.sin(p * f)) < 2e-5
    with pytest.raises(ValueError):
        Rotary(32, 700.0, 300, llama3={**sc, "low": 9.0})


def test_without_streams_the_stream_is_one_sum():
    """No ``streams``: no mixing tensors, the plain residual sum with the multiplier."""
    cfg = copy.deepcopy(U.CONFIGS["V"])
    del cfg["streams"]
    specs = build(cfg).param_specs()
    assert not any(".hc" in name for name in specs)
    assert "l0.norm1" in specs and build(cfg).spec.streams == 1


def test_plain_pieces():
    # the layer norm takes the mean off and has no offset
    x = torch.tensor([[1.0, 3.0]])
    assert torch.allclose(P.layer_norm(x, torch.tensor([2.0, 5.0]), 0.0), torch.tensor([[-2.0, 5.0]]))
    # streams: the mixing matrix is indexed [from, to], every part from the old ones
    xs = torch.tensor([[[1.0]], [[10.0]]])
    mix = torch.tensor([[1.0, 2.0], [3.0, 4.0]])
    new = P.update_streams(xs, torch.tensor([[100.0]]), mix, torch.tensor([1.0, 0.5]), 0.1)
    assert torch.allclose(new, torch.tensor([[[41.0]], [[47.0]]]))
    assert torch.allclose(P.read_streams(xs, torch.tensor([2.0, 0.5])), torch.tensor([[7.0]]))
    # one token: the bonus weighs its write, the decayed scan reads it as it is
    q = torch.tensor([[[1.0, 2.0]]])
    v = torch.tensor([[[3.0, 7.0]]])
    half = torch.full((1, 1, 2), 0.5)
    assert torch.allclose(P.decayed_scan(q, q, v, half), 5 * v)
    assert torch.allclose(P.bonus_scan(q, q, v, half, torch.tensor([[10.0, 1.0]])), 14 * v)
    # two tokens: the decayed scan's old write has decayed once, the bonus scan's has not
    two = lambda t: torch.cat([t, t])  # noqa: E731
    assert torch.allclose(P.decayed_scan(two(q), two(q), two(v), two(half))[1], 7.5 * v[0])
    assert torch.allclose(P.bonus_scan(two(q), two(q), two(v), two(half),
                                       torch.zeros(1, 2))[1], 5 * v[0])
    # halves turn, the rest passes
    t = P.rotate_halves(torch.tensor([[1.0, 0.0, 5.0], [1.0, 0.0, 5.0]]), [1.0])
    assert torch.allclose(t[1], torch.tensor([0.5403023, 0.8414710, 5.0]))
    # the router chooses with the correction and weighs without it
    w = {"router": torch.tensor([[0.0], [1.0], [-1.0]]), "correction": torch.tensor([0.0, -9.0, 9.0])}
    ids, wts = P.route(torch.ones(1, 1), w, {"experts": 3, "top": 2, "scale": 2.0})
    s = [1 / (1 + math.exp(-z)) for z in (-1.0, 0.0)]
    assert ids == [[2, 0]] and wts[0] == pytest.approx([2 * a / sum(s) for a in s])


@pytest.mark.parametrize("name", ["S", "V"])
def test_plain_model_is_causal_and_the_state_reaches_far(name):
    cfg = U.CONFIGS[name]
    tensors = U.random_tensors(cfg, 3)
    g = torch.Generator().manual_seed(0)
    toks = torch.randint(0, cfg["vocab"], (40,), generator=g).tolist()
    base = P.forward(cfg, tensors, toks)
    other = list(toks)
    other[10] = (other[10] + 1) % cfg["vocab"]
    changed = P.forward(cfg, tensors, other)
    assert torch.equal(changed[:10], base[:10])
    assert (changed[10:] - base[10:]).abs().amax(-1).min() > 1e-5
