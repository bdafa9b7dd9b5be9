"""Kumudra configurations drawn at random with fixed seeds (layer order, every size, head counts,
windows, rotations and their scaling, branch weights, decays, routers, layers without a feed-forward,
streams, loops, page sizes), each through a whole and a mixed trace in both precisions against the
plain implementation, free pages poisoned."""

import random

import pytest
import torch

import kumudra_util as U
import trace_util as T
from plain import kumudra_plain as P
from test_kumudra_model_gpu import compare, make_runner

pytestmark = pytest.mark.gpu


def draw_mlp(rng):
    kind = rng.random()
    if kind < 0.2:
        return None
    if kind < 0.5:
        return U.dense(rng.choice([8, 20, 64, 136]))
    experts = rng.randint(1, 10)
    return U.moe(rng.choice([8, 24, 40, 64]), experts, rng.randint(1, min(4, experts)),
                 rng.choice([1.0, 0.4, 2.5]))


def draw_layer(rng):
    kind = rng.choice(["parallel", "gla", "lightning"])
    heads = rng.choice([1, 2, 3, 4, 6])
    if kind == "gla":
        return U.gla(heads, rng.choice([4, 10, 16, 32, 48, 96]), rng.choice([6, 16, 40, 64, 72]),
                     rng.choice([1.0, 6.0, 16.0]), mlp=draw_mlp(rng))
    if kind == "lightning":
        return U.lightning(heads, rng.choice([4, 10, 16, 32, 64]), rng.choice([6, 16, 40, 64, 72]),
                           [rng.choice([0.0, 0.3, 0.9, 0.99, 1.0]) for _ in range(heads)],
                           mlp=draw_mlp(rng))
    # (a few head sizes, so that the attention kernels are compiled for few)
    top = rng.choice([16, 32, 48, 64, 128])
    dim, vdim = max(2, top - rng.randint(0, 15)), rng.randint(1, top)
    if rng.random() < 0.5 and vdim >= 2:
        dim, vdim = max(2, vdim), dim
    kv = rng.choice([1, 2, 3])
    scaled = rng.choice([None, U.scaling(rng.choice([2.0, 8.0]), 1.0, rng.choice([1.0, 4.0]),
                                         rng.choice([40, 300]))])
    att = U.left(kv * rng.choice([1, 2, 4]), kv, dim, vdim, rng.choice([1, 7, 16, 33, 64, 400]),
                 2 * rng.randint(1, dim // 2), base=rng.choice([30.0, 10000.0, 500000.0]),
                 scale=rng.choice([None, 0.07, 0.4]), scaled=scaled)
    return U.parallel(att, heads, rng.choice([4, 10, 16, 32, 48, 80]), rng.choice([1.0, 0.5, -0.8]),
                      rng.choice([1.0, 0.9, 0.0]), mlp=draw_mlp(rng))


def draw(seed):
    rng = random.Random(9000 + seed)
    layers = [draw_layer(rng) for _ in range(rng.randint(1, 4))]
    loop = None
    if rng.random() < 0.7:
        start = rng.randrange(len(layers))
        loop = (start, rng.randint(start, len(layers)), rng.choice([1, 2, 2, 3]))
    cfg = U.config(rng.choice([50, 128, 301]), rng.choice([32, 40, 64, 96, 128, 256]), layers,
                   streams=rng.choice([1, 2, 2, 3, 4, 6]), loop=loop,
                   eps=rng.choice([1e-5, 1e-6, 3e-4]), mult=rng.choice([1.0, 0.5, 0.8]),
                   scale=rng.choice([1.0, 0.3, 4.0]))
    lengths = [rng.randint(1, 140) for _ in range(5)] + [rng.choice([1, 2])]
    return cfg, lengths, rng.choice([8, 16, 32, 64])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(14))
def test_random_configuration(seed, dtype, tmp_path):
    from scratch_llm_b200.kernels import ops
    cfg, lengths, page = draw(seed)
    tensors = U.random_tensors(cfg, 700 + seed)
    folder = U.write_model(cfg, tensors, tmp_path / "m")
    reqs = T.make_requests(cfg["vocab"], lengths, seed=seed)
    want = {rid: P.forward(cfg, tensors, toks).float() for rid, toks in reqs.items()}
    for steps in (T.whole(reqs), T.mixed(reqs, seed=seed)):
        runner = make_runner(folder, dtype, page, T.peak_tokens(steps, round_to=max(64, page)),
                             max_requests=4, poison_free_pages=True)
        with torch.no_grad():
            got = T.run_in_process(runner, steps)
        ops.check_kernel_errors()
        assert len(got) == sum(lengths)
        compare(got, want, dtype)
