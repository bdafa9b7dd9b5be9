"""Small Kumudra configurations with random tensors of every kind (mixing weights of the streams,
decays that remember for long and for short, bonuses, token shifts, routers), written as model
folders, for the tests of that architecture."""

import torch

from nilevik_util import relative_error, write_model  # noqa: F401  (shared test helpers)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, scale=1.0):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "top": top, "scale": scale}}


def scaling(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def left(heads, kv_heads, dim, vdim, window, dims, base=10000.0, scale=None, scaled=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
            "scale": scale if scale is not None else dim ** -0.5, "mask": {"size": window},
            "rot": {"base": base, "dims": dims, "scaling": scaled}}


def parallel(att, heads, dim, left_scale=1.0, right_scale=1.0, mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": att, "right": {"heads": heads, "dim": dim}, "left_scale": left_scale,
        "right_scale": right_scale}}


def gla(heads, dim, vdim, tau=16.0, mlp=None):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim,
                                                 "tau": tau}}


def lightning(heads, dim, vdim, decay, mlp=None):
    return {"type": "lightning", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim,
                                                       "decay": list(decay)}}


def config(vocab, width, layers, streams=2, loop=None, eps=1e-5, mult=0.7, scale=0.5):
    cfg = {"architecture": "Kumudra", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "residual_mult": mult, "embedding": {"scale": scale}, "streams": streams,
           "layers": layers}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# Sizes differ from one configuration to the next in everything: each kind of mixer first, one to five
# streams, loops at the front, in the middle, over everything, of one pass and none at all, groups of
# one and of several query heads, values smaller and larger than keys, windows below, at and above a
# page and a tile, rotations of two entries and of the whole head, every branch of the frequency
# scaling and none, sizes in sixteens and sizes that are multiples of nothing, equal and unequal branch
# weights, layers without a feed-forward, dense ones, one expert and all of them, decays of 0 and 1.
CONFIGS = {
    "S": config(101, 48, [
        gla(3, 10, 6, 4.0, mlp=moe(24, 6, 2, 1.7)),
        parallel(left(4, 2, 12, 20, 13, 8, base=300.0, scaled=scaling(6.0, 1.0, 3.0, 90)), 3, 14,
                 0.6, 1.2, mlp=dense(40)),
        lightning(2, 9, 11, [0.4, 0.99], mlp=None)], streams=3, loop=(1, 3, 2), eps=1e-4),
    # rows of whole 16 bytes, sizes in sixteens: the chunk kernels of every scan, heads of 64 and of
    # 128 for the tensor-core attention
    "T": config(310, 128, [
        parallel(left(8, 2, 64, 48, 40, 64, base=200000.0, scale=0.11,
                      scaled=scaling(4.0, 0.5, 2.0, 300)), 4, 32, -0.8, 0.9,
                 mlp=moe(64, 9, 3, 0.8)),
        lightning(2, 64, 80, [0.2, 1.0], mlp=dense(96)),
        gla(2, 80, 96, 12.0, mlp=moe(40, 4, 4, 1.0)),
        parallel(left(3, 3, 96, 112, 150, 32), 2, 80, 1.0, 1.0, mlp=None)],
        streams=2, loop=(1, 3, 2), eps=3e-6, mult=0.5, scale=1.0),
    "U": config(131, 64, [
        lightning(4, 16, 136, [0.0, 0.5, 0.97, 1.0], mlp=dense(24)),
        parallel(left(2, 1, 32, 16, 1, 2, scale=0.4), 1, 40, 1.3, 0.0, mlp=moe(32, 1, 1, 2.5)),
        gla(1, 144, 24, 1.0, mlp=None)], streams=5, eps=1e-6, mult=0.4, scale=2.0),
    "V": config(90, 40, [
        parallel(left(5, 5, 8, 8, 64, 8, base=50.0), 5, 8, 0.5, -0.5, mlp=dense(33)),
        gla(5, 8, 8, 8.0, mlp=moe(17, 3, 1, 1.1))], streams=1, loop=(1, 2, 3)),
}


def random_tensors(cfg, seed):
    """{name: tensor} for every tensor of the architecture, as bfloat16-exact values in 32-bit
    (so that both precisions and the plain model hold the same numbers)."""
    g = torch.Generator().manual_seed(seed)

    def normal(shape, std=1.0, mean=0.0):
        t = torch.randn(shape, generator=g) * std + mean
        return t.to(torch.bfloat16).float()

    d, V, s = cfg["width"], cfg["vocab"], cfg["streams"]
    t = {"embed": normal((V, d)), "final.norm": normal((d,), 0.2, 1.0)}
    for i, one in enumerate(cfg["layers"]):
        m, p = one["mixer"], f"l{i}."
        for q in ("1", "2")[:1 if one["mlp"] is None else 2]:
            t[p + "norm" + q] = normal((d,), 0.2, 1.0)
            t[p + f"hc{q}.in"] = normal((s,), 0.4, 1.0 / s)
            t[p + f"hc{q}.out"] = normal((s,), 0.3, 0.8)
            t[p + f"hc{q}.mix"] = (0.8 * torch.eye(s) + normal((s, s), 0.15)).bfloat16().float()
        if one["type"] == "parallel":
            a, r = m["left"], m["right"]
            H, G, hd = a["heads"], a["kv_heads"], r["heads"] * r["dim"]
            for name, rows in (("q", H * a["dim"]), ("k", G * a["dim"]), ("v", G * a["vdim"])):
                t[p + f"mix.left.{name}"] = normal((rows, d), d ** -0.5)
                t[p + f"mix.left.{name}.b"] = normal((rows,), 0.4)
            t[p + "mix.left.o"] = normal((d, H * a["vdim"]), (H * a["vdim"]) ** -0.5)
            rank = 5 + 3 * i
            for name in "rkvgw":
                t[p + f"mix.right.mu.{name}"] = normal((d,), 0.4, 0.5)
            for name in "rkvg":
                t[p + f"mix.right.{name}"] = normal((hd, d), d ** -0.5)
            t[p + "mix.right.w1"] = normal((rank, d), d ** -0.5)
            t[p + "mix.right.w2"] = normal((hd, rank), rank ** -0.5)
            # decays from a few tokens' memory to hundreds', some channels that keep next to nothing
            t[p + "mix.right.w0"] = normal((hd,), 2.0, -2.5)
            t[p + "mix.right.u"] = normal((r["heads"], r["dim"]), 0.7, 0.5)
            t[p + "mix.right.norm"] = normal((hd,), 0.2, 1.0)
            t[p + "mix.right.o"] = normal((d, hd), hd ** -0.5)
        else:
            H, hk, hv = m["heads"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for name, rows in (("q", hk), ("k", hk), ("v", hv), ("g", hv)):
                t[p + f"mix.{name}"] = normal((rows, d), d ** -0.5)
            t[p + "mix.o"] = normal((d, hv), hv ** -0.5)
            if one["type"] == "gla":
                rank = 4 + 5 * i
                t[p + "mix.a1"] = normal((rank, d), d ** -0.5)
                t[p + "mix.a2"] = normal((hk, rank), 2.0 * rank ** -0.5)
                t[p + "mix.a2.b"] = normal((hk,), 2.0, 1.0)
            t[p + "mix.norm"] = normal((m["vdim"] if one["type"] == "gla" else hv,), 0.2, 1.0)
        mlp = one["mlp"]
        if mlp is None:
            continue
        sizes = {"mlp": mlp["ff"]} if mlp["kind"] == "dense" else \
            {f"mlp.e{e}": mlp["expert"]["ff"] for e in range(mlp["router"]["experts"])}
        if mlp["kind"] == "moe":
            t[p + "mlp.router"] = normal((len(sizes), d), 2.0 * d ** -0.5)
            t[p + "mlp.correction"] = normal((len(sizes),), 0.3)
        for name, ff in sizes.items():
            t[p + f"{name}.gate"] = normal((ff, d), d ** -0.5)
            t[p + f"{name}.up"] = normal((ff, d), d ** -0.5)
            t[p + f"{name}.down"] = normal((d, ff), ff ** -0.5)
    return t
