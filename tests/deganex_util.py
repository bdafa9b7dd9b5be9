"""Small Deganex configurations with random tensors of every kind (state-space and matrix-memory
gates that remember for long and for short, latent projections, gates, routers, shared experts,
the pair table), written as model folders, for the tests of that architecture."""

import math

import torch

from nilevik_util import relative_error, write_model  # noqa: F401  (shared test helpers)


def latent(heads, dim, rot_dim, vdim, kv_rank, base=10000.0, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
        "scale": scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim),
        "rot": {"base": base, "dims": rot_dim}}}


def mlstm(heads, dim, vdim, gate_cap=8.0, mlp=None):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim,
                                                   "gate_cap": gate_cap}}


def mamba2(heads, vdim, state, groups, conv, norm_groups, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {
        "heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
        "norm_groups": norm_groups}}


def moe(ff, experts, top, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def again(layers, j):
    """Layer j of ``layers`` once more, with its tensors."""
    return dict(layers[j], weights_of=j)


def config(vocab, width, layers, bigram=(61, 7, 3), eps=1e-5, softcap=9.0):
    cfg = {"architecture": "Deganex", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "logit_softcap": softcap, "layers": layers}
    if bigram is not None:
        cfg["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    return cfg


def _with_again(layers, *which):
    return layers + [again(layers, j) for j in which]


# Sizes differ from one configuration to the next in everything: each kind of mixer first, layers
# that run once and twice, head counts from 1 to 6, value sizes smaller and larger than key sizes
# and beyond 64, groups of 1 and of every head, one to four convolution taps, one norm part and as
# many as do not line up with the heads, cached vectors that are and are not a
# multiple of 16 (and of 64), layers without a feed-forward, without a shared expert, one choice
# and all of them, tables of one and of many buckets, multipliers of 0 and larger than the table,
# with and without caps.
CONFIGS = {
    "S": config(97, 48, _with_again(
        [mlstm(3, 6, 10, 4.0, mlp=moe(24, 6, 2, shared=40)),
         mamba2(4, 10, 12, 2, 3, 5, mlp=moe(40, 5, 1)),
         latent(3, 8, 4, 10, 21, base=500.0, scale=0.4, mlp=None),
         latent(5, 12, 6, 6, 20, base=30.0, mlp=moe(16, 3, 3, shared=8))], 1, 0, 2),
        bigram=(61, 7, 3), eps=1e-4, softcap=6.0),
    # rows of whole 16 bytes, key sizes in sixteens: the chunk kernels, cached vectors of 128 and
    # of 64 entries for the tensor-core attention
    "T": config(300, 128, _with_again(
        [latent(6, 24, 32, 40, 96, base=150000.0, mlp=moe(64, 9, 3, shared=128)),
         mamba2(6, 24, 32, 1, 4, 1, mlp=moe(40, 4, 2, shared=64)),
         mlstm(2, 48, 72, 12.0, mlp=moe(64, 6, 2)),
         latent(4, 64, 16, 64, 48, base=300.0, mlp=None)], 1, 2, 3),
        bigram=(503, 911, 5000), eps=1e-6, softcap=20.0),
    "U": config(131, 64, _with_again(
        [mamba2(2, 40, 16, 2, 1, 2, mlp=None),
         mlstm(1, 16, 136, 30.0, mlp=moe(32, 4, 4, shared=16)),
         mamba2(3, 16, 80, 3, 2, 3, mlp=moe(24, 8, 3, shared=24))], 0, 1),
        bigram=(1, 0, 1), eps=3e-6, softcap=0.0),
}


def random_tensors(cfg, seed):
    """{name: tensor} for every tensor of the architecture, as bfloat16-exact values in 32-bit
    (so that both precisions and the plain model hold the same numbers)."""
    g = torch.Generator().manual_seed(seed)

    def normal(shape, std=1.0, mean=0.0):
        t = torch.randn(shape, generator=g) * std + mean
        return t.to(torch.bfloat16).float()

    d, V = cfg["width"], cfg["vocab"]
    t = {"embed": normal((V, d)), "head": normal((V, d), 3.0 * d ** -0.5),
         "final.norm": normal((d,), 0.2, 1.0)}
    bigram = (cfg.get("embedding") or {}).get("bigram")
    if bigram is not None:
        t["bigram"] = normal((bigram["buckets"] + 1, d))
    for i, one in enumerate(cfg["layers"]):
        if one.get("weights_of") is not None:
            continue
        m, p = one["mixer"], f"l{i}."
        t[p + "norm1"] = normal((d,), 0.2, 1.0)
        H, dv = m["heads"], m["vdim"]
        t[p + "mix.o"] = normal((d, H * dv), (H * dv) ** -0.5)
        if one["type"] == "latent_attention":
            dim, r, R = m["dim"], m["rot_dim"], m["kv_rank"]
            t[p + "mix.q"] = normal((H * (dim + r), d), d ** -0.5)
            t[p + "mix.dkv"] = normal((R + r, d), d ** -0.5)
            t[p + "mix.dkv.norm"] = normal((R,), 0.2, 1.0)
            t[p + "mix.uk"] = normal((H * dim, R), R ** -0.5)
            t[p + "mix.uv"] = normal((H * dv, R), R ** -0.5)
            t[p + "mix.g"] = normal((H * dv, d), 2.0 * d ** -0.5)
        elif one["type"] == "mlstm":
            D = m["dim"]
            for name, rows in (("q", H * D), ("k", H * D), ("v", H * dv), ("g", H * dv)):
                t[p + f"mix.{name}"] = normal((rows, d), d ** -0.5)
            t[p + "mix.norm"] = normal((H * dv,), 0.2, 1.0)
            # input gates of both signs; forget gates from a few tokens' memory to hundreds'
            t[p + "mix.i"] = normal((H, d), 2.0 * d ** -0.5)
            t[p + "mix.i.b"] = normal((H,), 1.0, -1.0)
            t[p + "mix.f"] = normal((H, d), d ** -0.5)
            t[p + "mix.f.b"] = normal((H,), 1.5, 4.0)
        else:
            N, G = m["state"], m["groups"]
            inner, C = H * dv, H * dv + 2 * G * N
            t[p + "mix.in"] = normal((inner + C + H, d), d ** -0.5)
            t[p + "mix.conv"] = normal((C, m["conv"]), m["conv"] ** -0.5)
            t[p + "mix.conv.b"] = normal((C,), 0.3)
            # step sizes from a hundredth to one, rates likewise from slow to fast
            t[p + "mix.dt_bias"] = normal((H,), 1.0, -2.0)
            t[p + "mix.A_log"] = normal((H,), 1.5, -1.0)
            t[p + "mix.D"] = normal((H,), 0.5, 0.5)
            t[p + "mix.norm"] = normal((inner,), 0.2, 1.0)
        mlp = one["mlp"]
        if mlp is None:
            continue
        t[p + "norm2"] = normal((d,), 0.2, 1.0)
        E, f = mlp["router"]["experts"], mlp["expert"]["ff"]
        t[p + "mlp.router"] = normal((E, d), 2.0 * d ** -0.5)
        sizes = {f"e{e}": f for e in range(E)}
        if mlp.get("shared") is not None:
            sizes["shared"] = mlp["shared"]["ff"]
            t[p + "mlp.shared.sg"] = normal((1, d), 2.0 * d ** -0.5)
        for name, width in sizes.items():
            t[p + f"mlp.{name}.gate"] = normal((width, d), d ** -0.5)
            t[p + f"mlp.{name}.up"] = normal((width, d), d ** -0.5)
            t[p + f"mlp.{name}.down"] = normal((d, width), width ** -0.5)
    return t
