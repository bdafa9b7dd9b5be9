"""The Deganex configuration without a GPU: config.json keys to layers as data, tensor names,
layers that run again with a state of their own, what the configuration refuses, and the plain
implementation's own properties."""

import json

import pytest
import torch

import deganex_util as U
from plain import deganex_plain as P


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
        assert tuple(tensors[key].shape) == tuple(spec.shape), key


def test_a_layer_that_runs_again_has_no_tensors_and_a_state_of_its_own():
    model = build(U.CONFIGS["S"])
    assert [(r.layer, r.cache, r.write) for r in model.spec.order] == \
        [(0, 0, True), (1, 1, True), (2, 2, True), (3, 3, True), (1, 4, True), (0, 5, True),
         (2, 6, True)]
    assert len(model.blocks) == 4
    assert not any(n.startswith(("l4.", "l5.", "l6.")) for n in model.param_specs())
    kv, st = model.cache_specs()
    assert len(kv) == len(st) == 8                       # the last: the previous token
    assert [k is not None for k in kv] == [False, False, True, True, False, False, True, False]
    assert kv[2] == kv[6] and kv[2].planes == 1 and kv[2].head_dim == 32     # 21 + 4, in sixteens
    # the matrix memory: the value columns and the normaliser, and a running maximum per head
    assert [tuple(s.shape) for s in st[0]] == [(3, 11, 6), (3,)] == [tuple(s.shape) for s in st[5]]
    assert [tuple(s.shape) for s in st[1]] == [(4, 10, 12), (2, 4 * 10 + 2 * 2 * 12)]
    assert st[2] is None and st[7].shape == () and st[7].dtype == torch.int32
    one_tap = build(U.CONFIGS["U"]).cache_specs()[1][0]
    assert tuple(one_tap.shape) == (2, 40, 16)           # one tap: nothing to carry beside S


def test_layers_may_lead_to_their_owner_over_another_and_come_before_it():
    layers = [U.mlstm(2, 8, 8, mlp=None), U.mamba2(2, 8, 8, 1, 2, 1)]
    cfg = U.config(50, 32, layers + [U.again(layers, 1), dict(layers[1], weights_of=2)])
    assert [r.layer for r in build(cfg).spec.order] == [0, 1, 1, 1]
    cfg = U.config(50, 32, [dict(layers[1], weights_of=1), layers[1]])
    assert [r.layer for r in build(cfg).spec.order] == [0, 0]
    assert "l1.mix.in" in build(cfg).param_specs()


def test_round_trip_and_refusals():
    from scratch_llm_b200.config import DeganexConfig, config_from_dict
    for name in U.CONFIGS:
        cfg = config_from_dict(U.CONFIGS[name])
        assert isinstance(cfg, DeganexConfig)
        again = config_from_dict(cfg.to_dict())
        assert again == cfg and again.model_spec() == cfg.model_spec()

    def broken(change):
        c = json.loads(json.dumps(U.CONFIGS["S"]))   # (layers that run again share nothing)
        change(c)
        return c

    bad = [lambda c: c["layers"][4].update(weights_of=4),                   # itself
           lambda c: c["layers"][4].update(weights_of=8),                   # nobody
           lambda c: c["layers"][4].update(weights_of=0),                   # another kind
           lambda c: c["layers"][4]["mixer"].update(state=16),              # another size
           lambda c: (c["layers"][1].update(weights_of=4)),                 # a circle
           lambda c: c["layers"][0].update(type="attention"),
           lambda c: c["layers"][0]["mixer"].update(gate_cap=0.0),
           lambda c: c["layers"][2]["mixer"]["rot"].update(dims=5),
           lambda c: c["layers"][2]["mixer"].pop("scale"),
           lambda c: c["layers"][1]["mixer"].update(groups=3),
           lambda c: c["layers"][1]["mixer"].update(norm_groups=3),
           lambda c: c["layers"][0]["mlp"].update(kind="dense"),
           lambda c: c["layers"][0]["mlp"]["router"].update(top=7),
           lambda c: c["embedding"]["bigram"].update(buckets=0),
           lambda c: c["embedding"]["bigram"].update(mul_prev=-1),
           lambda c: c.update(logit_softcap=-1.0),
           lambda c: c.pop("norm")]
    for change in bad:
        with pytest.raises(ValueError):
            config_from_dict(broken(change))


def test_plain_pieces():
    # pairs: the last row first, then the hash of (previous, current)
    assert P.bigram_rows([5, 6, 5], {"buckets": 10, "mul_prev": 3, "mul_cur": 4}) == [10, 9, 8]
    # one token of the matrix memory: S = k v^T with weight 1 (the gate's maximum is its own), n = k
    q = k = torch.tensor([[[1.0, 2.0]]], dtype=torch.float64)
    v = torch.tensor([[[3.0, 7.0]]], dtype=torch.float64)
    big = torch.full((1, 1), 4.0, dtype=torch.float64)
    assert torch.allclose(P.mlstm_scan(q, k, v, big, -big), v, rtol=1e-6)       # 5 v / (5 + 1e-6)
    # a weak input gate: m stays f + 0, the floor exp(-m) wins over |n . q|
    out = P.mlstm_scan(q, k, v, -big, torch.zeros(1, 1, dtype=torch.float64))
    assert torch.allclose(out, 5 * v * torch.exp(-big) / (1 + 1e-6))
    # the state-space rule sees its own token: y = dt (B . C) x + D x
    one = torch.ones((1, 1), dtype=torch.float64)
    y = P.ssd_scan(v, k, q, 0.5 * one, one[0], 2.0 * one[0])
    assert torch.allclose(y, v * (0.5 * 5 + 2.0))
    # the convolution's last tap meets the current token, the bias is there from the start
    x = torch.arange(1.0, 5.0)[:, None]
    taps = torch.tensor([[100.0, 10.0, 1.0]])
    assert P.short_conv(x, taps, torch.tensor([0.5]))[:, 0].tolist() == [1.5, 12.5, 123.5, 234.5]
    # parts are normed one by one
    z = P.grouped_norm(torch.tensor([[3.0, 4.0, 30.0, 40.0]]), 2, torch.ones(4), 0.0)
    assert torch.allclose(z[0, :2], z[0, 2:])
    # adjacent pairs turn
    t = P.rotate_pairs(torch.tensor([[1.0, 0.0, 5.0], [1.0, 0.0, 5.0]]), 2, 10.0)
    assert torch.allclose(t[1], torch.tensor([0.5403023, 0.8414710, 5.0]))


def test_plain_model_is_causal_and_remembers_the_previous_token():
    cfg = U.CONFIGS["S"]
    tensors = U.random_tensors(cfg, 3)
    g = torch.Generator().manual_seed(0)
    toks = torch.randint(0, cfg["vocab"], (30,), generator=g).tolist()
    base = P.forward(cfg, tensors, toks)
    other = list(toks)
    other[20] = (other[20] + 1) % cfg["vocab"]
    changed = P.forward(cfg, tensors, other)
    assert torch.equal(changed[:20], base[:20])
    assert (changed[20:] - base[20:]).abs().amax(-1).min() > 1e-4
