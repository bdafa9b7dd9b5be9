"""Deganex configurations drawn at random with fixed seeds (every size, head counts and groups,
taps, norm parts, gate caps, latent sizes, routers with and without a shared expert, layers without a
feed-forward, layers that run again, pair tables, page sizes), each through a whole and a mixed
trace in both precisions against the plain implementation, free pages poisoned."""

import random

import pytest
import torch

import deganex_util as U
import trace_util as T
from plain import deganex_plain as P
from test_deganex_model_gpu import compare, make_runner

pytestmark = pytest.mark.gpu


def draw_mlp(rng):
    if rng.random() < 0.25:
        return None
    experts = rng.randint(1, 10)
    return U.moe(rng.choice([8, 24, 40, 64, 136]), experts, rng.randint(1, min(4, experts)),
                 shared=rng.choice([None, 8, 24, 72]))


def draw_layer(rng):
    kind = rng.choice(["latent", "mlstm", "mamba2"])
    if kind == "latent":
        # the cached vector (latent, rotated part, zeros up to a multiple of 16) has one of a few
        # sizes, so that the attention kernels are compiled for few
        cached = rng.choice([16, 32, 48, 64, 80, 128, 192, 256, 288])
        rot_dim = 2 * rng.randint(1, min(24, cached // 2 - 1))
        return U.latent(rng.choice([1, 2, 3, 4, 8, 12]), rng.choice([4, 8, 16, 24, 32, 64]),
                        rot_dim, rng.choice([8, 16, 24, 48, 64]),
                        max(1, cached - rot_dim - rng.randint(0, 15)),
                        base=rng.choice([30.0, 10000.0, 200000.0]),
                        scale=rng.choice([None, 0.05, 0.3]), mlp=draw_mlp(rng))
    if kind == "mlstm":
        return U.mlstm(rng.choice([1, 2, 3, 6]), rng.choice([4, 10, 16, 32, 48, 96]),
                       rng.choice([6, 16, 40, 64, 72]), rng.choice([2.0, 8.0, 25.0]),
                       mlp=draw_mlp(rng))
    groups = rng.choice([1, 2, 3])
    heads = groups * rng.choice([1, 2, 4])
    vdim = rng.choice([8, 10, 24, 64, 72])
    parts = rng.choice([p for p in (1, 2, heads, 2 * heads) if (heads * vdim) % p == 0])
    return U.mamba2(heads, vdim, rng.choice([6, 16, 32, 64, 112]), groups, rng.randint(1, 5), parts,
                    mlp=draw_mlp(rng))


def draw(seed):
    rng = random.Random(6000 + seed)
    layers = [draw_layer(rng) for _ in range(rng.randint(1, 5))]
    # (at most eight layer runs: bfloat16 is compared with an exact model, and every routed
    # layer on the way may take another expert for a token whose logits are close)
    layers += [U.again(layers, rng.randrange(len(layers))) for _ in range(rng.randint(0, 3))]
    bigram = rng.choice([None, (1, 1, 1), (rng.randint(2, 400), rng.randint(0, 99),
                                           rng.randint(0, 99))])
    cfg = U.config(rng.choice([50, 128, 301]), rng.choice([32, 40, 64, 96, 128, 256]), layers,
                   bigram=bigram, eps=rng.choice([1e-5, 1e-6, 3e-4]),
                   softcap=rng.choice([0.0, 5.0, 30.0]))
    lengths = [rng.randint(1, 140) for _ in range(5)] + [rng.choice([1, 2])]
    return cfg, lengths, rng.choice([8, 16, 32, 64])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(12))
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
