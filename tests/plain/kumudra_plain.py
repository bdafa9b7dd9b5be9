"""A plain, slow Kumudra: whole sequences, no cache, 64-bit, one function per mechanism.  It
shares no code with the package; the tests compare the engine with it.

``w`` maps tensor names to 64-bit tensors; a mixer's and a feed-forward's functions take the
tensors below their own prefix (``q``, ``left.q.b``, ..., ``router``, ``e0.up``, ...).  ``h``
[T, width] is what the norm in front of the branch left.
"""

import math

import torch


# ------------------------------------------------------------------------------ small pieces

def layer_norm(x, gain, eps):
    mean = x.mean(-1, keepdim=True)
    dev = x - mean
    return dev / torch.sqrt(dev.pow(2).mean(-1, keepdim=True) + eps) * gain


def rms_unit(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return torch.clamp(z, max=0) - torch.log1p(torch.exp(-z.abs()))


def below(w, prefix):
    return {k[len(prefix) + 1:]: v for k, v in w.items() if k.startswith(prefix + ".")}


# ---------------------------------------------------------------------------------- streams

def read_streams(xs, weights):
    """xs [s, T, width] -> [T, width]"""
    return sum(weights[s] * xs[s] for s in range(xs.shape[0]))


def update_streams(xs, y, mix, out, mult):
    """Every stream from all old ones (mix is [from, to]) and its share of the sublayer's
    output."""
    n = xs.shape[0]
    return torch.stack([sum(mix[s, t] * xs[s] for s in range(n)) + mult * out[t] * y
                        for t in range(n)])


# -------------------------------------------------------------------------------- attention

def frequencies(rot):
    """One frequency per pair; the long ones slowed down by a factor, with a ramp between."""
    sc = rot.get("scaling")
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if sc is not None:
            wavelength = 2 * math.pi / f
            if wavelength < sc["original"] / sc["high"]:
                pass
            elif wavelength > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            else:
                s = (sc["original"] / wavelength - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_halves(v, freqs):
    """v: [T, ..., n] at positions 0 .. T-1; entry i turns with entry i + len(freqs), the entries
    from 2 len(freqs) on pass."""
    out = v.clone()
    half = len(freqs)
    for p in range(v.shape[0]):
        for i, f in enumerate(freqs):
            c, s = math.cos(p * f), math.sin(p * f)
            x, y = v[p, ..., i], v[p, ..., i + half]
            out[p, ..., i] = x * c - y * s
            out[p, ..., i + half] = y * c + x * s
    return out


def window_attention(h, w, m):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    f = frequencies(m["rot"])
    q = rotate_halves((h @ w["q"].T + w["q.b"]).view(T, H, d), f)
    k = rotate_halves((h @ w["k"].T + w["k.b"]).view(T, G, d), f)
    v = (h @ w["v"].T + w["v.b"]).view(T, G, dv)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) & (i - j < m["mask"]["size"])
    out = torch.zeros((T, H, dv), dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].T * m["scale"]).masked_fill(~seen, -math.inf)
        out[:, head] = torch.softmax(s, -1) @ v[:, g]
    return out.reshape(T, H * dv) @ w["o"].T


# ------------------------------------------------------------------------------- time mixing

def shifted(h):
    """The previous token's h, zeros for the first."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def bonus_scan(r, k, v, decay, u):
    """r, k, decay: [T, H, D], v: [T, H, V], u: [H, D] -> o [T, H, V]: the read-out sees the old
    state and the token's own write weighted by u."""
    T, H, D = r.shape
    S = torch.zeros((H, D, v.shape[2]), dtype=r.dtype)
    out = torch.zeros((T, H, v.shape[2]), dtype=r.dtype)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S + u[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    return out


def time_mixing(h, w, m, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    prev = shifted(h)

    def mix(name):
        return h + (prev - h) * w["mu." + name]

    r, k, v = ((mix(n) @ w[n].T).view(T, H, D) for n in "rkv")
    gate = silu(mix("g") @ w["g"].T)
    z = torch.tanh(mix("w") @ w["w1"].T) @ w["w2"].T + w["w0"]
    decay = torch.exp(-torch.exp(z)).view(T, H, D)
    o = rms_unit(bonus_scan(r, k, v, decay, w["u"]), eps).reshape(T, H * D)
    return (o * w["norm"] * gate) @ w["o"].T


def parallel(h, w, m, eps):
    return m["left_scale"] * window_attention(h, below(w, "left"), m["left"]) \
        + m["right_scale"] * time_mixing(h, below(w, "right"), m["right"], eps)


# ------------------------------------------------------------------------- linear attention

def decayed_scan(q, k, v, decay):
    """q, k, decay: [T, H, D], v: [T, H, V] -> o [T, H, V]: the read-out sees the new state."""
    T, H, D = q.shape
    S = torch.zeros((H, D, v.shape[2]), dtype=q.dtype)
    out = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def gla(h, w, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w["k"].T).view(T, H, D)
    v = (h @ w["v"].T).view(T, H, V)
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    alpha = torch.exp(log_sigmoid(z) / m["tau"]).view(T, H, D)
    o = (rms_unit(decayed_scan(q, k, v, alpha), eps) * w["norm"]).reshape(T, H * V)
    return (o * silu(h @ w["g"].T)) @ w["o"].T


def lightning(h, w, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w["q"].T).view(T, H, D)
    k = silu(h @ w["k"].T).view(T, H, D)
    v = silu(h @ w["v"].T).view(T, H, V)
    decay = torch.tensor(m["decay"], dtype=h.dtype)[None, :, None].expand(T, H, D)
    o = decayed_scan(q, k, v, decay).reshape(T, H * V)
    return (rms_unit(o, eps) * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


# ------------------------------------------------------------------------------ feed-forward

def gated_ff(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(h, w, router):
    """(chosen experts per token, best first; their weights)."""
    s = sigmoid(h @ w["router"].T)
    choice = s + w["correction"]
    chosen, weights = [], []
    for t in range(h.shape[0]):
        ids = sorted(range(router["experts"]), key=lambda e: (-float(choice[t, e]), e))
        ids = ids[:router["top"]]
        total = sum(float(s[t, e]) for e in ids) + 1e-20
        chosen.append(ids)
        weights.append([float(s[t, e]) / total * router["scale"] for e in ids])
    return chosen, weights


def moe_ff(h, w, mlp):
    chosen, weights = route(h, w, mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in zip(chosen[t], weights[t]):
            out[t] += weight * gated_ff(h[t:t + 1], below(w, f"e{e}"))[0]
    return out


def feed_forward(h, w, mlp):
    return gated_ff(h, w) if mlp["kind"] == "dense" else moe_ff(h, w, mlp)


# ------------------------------------------------------------------------------------ the model

MIXERS = {"parallel": parallel, "gla": gla, "lightning": lightning}


def run_order(cfg):
    """Layer of every run."""
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    n = len(cfg["layers"])
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] \
        + list(range(loop["stop"], n))


def forward(cfg, tensors, tokens, streams=None):
    """Logits [T, vocab] of one whole sequence; ``streams`` (a list) receives the sum of the
    residual streams after every layer run."""
    w = {k: v.double() for k, v in tensors.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][[int(t) for t in tokens]] * cfg["embedding"]["scale"]
    xs = torch.stack([x] * cfg["streams"])
    for i in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}"
        subs = [("1", lambda h: MIXERS[layer["type"]](h, below(w, p + ".mix"), layer["mixer"], eps))]
        if layer.get("mlp") is not None:
            subs.append(("2", lambda h: feed_forward(h, below(w, p + ".mlp"), layer["mlp"])))
        for q, sub in subs:
            hc = below(w, f"{p}.hc{q}")
            y = sub(layer_norm(read_streams(xs, hc["in"]), w[f"{p}.norm{q}"], eps))
            xs = update_streams(xs, y, hc["mix"], hc["out"], mult)
        if streams is not None:
            streams.append(xs.sum(0))
    return layer_norm(xs.sum(0), w["final.norm"], eps) @ w["embed"].T
