"""A plain, slow Deganex: whole sequences, no cache, 64-bit, one function per mechanism.  It
shares no code with the package; the tests compare the engine with it.

``w`` maps tensor names to 64-bit tensors; a mixer's and a feed-forward's functions take the
tensors below their own prefix (``q``, ``dkv``, ..., ``router``, ``e0.up``, ...).  ``h`` [T, width]
is what the norm in front of the branch left.
"""

import math

import torch

DIVISOR_FLOOR = 1e-6       # added to the matrix memory's divisor


# ------------------------------------------------------------------------------ small pieces

def rms_unit(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def rms_norm(x, gain, eps):
    return rms_unit(x, eps) * gain


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rotate_pairs(v, dims, base):
    """v: [T, ..., n] at positions 0 .. T-1; of the first ``dims`` entries, entry 2i turns with
    entry 2i + 1 by the angle position * base^(-2i / dims); the rest pass."""
    out = v.clone()
    for p in range(v.shape[0]):
        for i in range(dims // 2):
            a = p * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            x, y = v[p, ..., 2 * i], v[p, ..., 2 * i + 1]
            out[p, ..., 2 * i] = x * c - y * s
            out[p, ..., 2 * i + 1] = y * c + x * s
    return out


# --------------------------------------------------------------------------------- embedding

def bigram_rows(tokens, bigram):
    """The row of the bigram table that each token of a sequence adds."""
    rows = []
    for t, tok in enumerate(tokens):
        if t == 0:
            rows.append(bigram["buckets"])
        else:
            rows.append((tokens[t - 1] * bigram["mul_prev"] + tok * bigram["mul_cur"])
                        % bigram["buckets"])
    return rows


# -------------------------------------------------------------------------- latent attention

def latent_attention(h, w, m, eps):
    """Keys and values per head are formed from the latent, as the definition has them (not
    absorbed into the queries)."""
    T = h.shape[0]
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m["rot"]
    q = (h @ w["q"].T).view(T, H, d + r)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :R], w["dkv.norm"], eps)
    k_rot = rotate_pairs(down[:, R:], rot["dims"], rot["base"])              # [T, r]
    q_rot = rotate_pairs(q[..., d:], rot["dims"], rot["base"])               # [T, H, r]
    k = (c @ w["uk"].T).view(T, H, d)
    v = (c @ w["uv"].T).view(T, H, dv)
    out = torch.zeros((T, H, dv), dtype=h.dtype)
    for head in range(H):
        s = (q[:, head, :d] @ k[:, head].T + q_rot[:, head] @ k_rot.T) * m["scale"]
        s = s.masked_fill(torch.ones(T, T).triu(1).bool(), -math.inf)
        out[:, head] = torch.softmax(s, -1) @ v[:, head]
    return (out.reshape(T, H * dv) * sigmoid(h @ w["g"].T)) @ w["o"].T


# ------------------------------------------------------------------------------ matrix memory

def mlstm_gates(h, w, cap):
    """(log input gate, log forget gate), each [T, H]."""
    i = cap * torch.tanh((h @ w["i"].T + w["i.b"]) / cap)
    f = -softplus(-(cap * torch.tanh((h @ w["f"].T + w["f.b"]) / cap)))
    return i, f


def mlstm_scan(q, k, v, i, f):
    """q, k: [T, H, D], v: [T, H, V], i, f: [T, H] -> o [T, H, V]."""
    T, H, D = q.shape
    V = v.shape[2]
    S = torch.zeros((H, D, V), dtype=q.dtype)
    n = torch.zeros((H, D), dtype=q.dtype)
    m = torch.zeros((H,), dtype=q.dtype)
    out = torch.zeros((T, H, V), dtype=q.dtype)
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        m = m_new
        read = torch.einsum("hdv,hd->hv", S, q[t])
        div = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + DIVISOR_FLOOR
        out[t] = read / div[:, None]
    return out


def mlstm(h, w, m, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w["k"].T).view(T, H, D)
    v = (h @ w["v"].T).view(T, H, V)
    i, f = mlstm_gates(h, w, m["gate_cap"])
    o = rms_unit(mlstm_scan(q, k, v, i, f), eps).reshape(T, H * V)
    return (o * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


# ------------------------------------------------------------------- state-space recurrence

def short_conv(x, taps, bias):
    """Causal convolution over time per channel: ``x`` [T, C], ``taps`` [C, K] whose last
    column meets the current token; zeros before the start."""
    K = taps.shape[1]
    out = bias.expand_as(x).clone()
    for t in range(x.shape[0]):
        for j in range(K):
            src = t - (K - 1 - j)
            if src >= 0:
                out[t] = out[t] + taps[:, j] * x[src]
    return out


def ssd_scan(x, B, C, dt, rate, D):
    """x: [T, H, V], B, C: [T, G, N], dt: [T, H], rate (exp of A_log) and D: [H] -> y [T, H, V]."""
    T, H, V = x.shape
    G, N = B.shape[1:]
    group = torch.arange(H) // (H // G)
    S = torch.zeros((H, N, V), dtype=x.dtype)
    y = torch.zeros((T, H, V), dtype=x.dtype)
    for t in range(T):
        b, c = B[t][group], C[t][group]
        S = torch.exp(-rate * dt[t])[:, None, None] * S \
            + dt[t][:, None, None] * b[:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnv,hn->hv", S, c) + D[:, None] * x[t]
    return y


def grouped_norm(y, groups, gain, eps):
    """Each of ``groups`` equal parts over its own root mean square."""
    T = y.shape[0]
    return rms_unit(y.view(T, groups, -1), eps).reshape(T, -1) * gain


def mamba2(h, w, m, eps):
    T = h.shape[0]
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, gn = H * V, G * N
    proj = h @ w["in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * gn], proj[:, 2 * inner + 2 * gn:]
    xbc = silu(short_conv(xbc, w["conv"], w["conv.b"]))
    x = xbc[:, :inner].view(T, H, V)
    B = xbc[:, inner:inner + gn].view(T, G, N)
    C = xbc[:, inner + gn:].view(T, G, N)
    y = ssd_scan(x, B, C, softplus(dt + w["dt_bias"]), torch.exp(w["A_log"]), w["D"])
    y = y.reshape(T, inner) * silu(z)
    return grouped_norm(y, m["norm_groups"], w["norm"], eps) @ w["o"].T


# ------------------------------------------------------------------------------- feed-forward

def gated_ff(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(h, w, router):
    """(chosen experts per token, best first; their weights)."""
    z = h @ w["router"].T
    chosen, weights = [], []
    for t in range(h.shape[0]):
        ids = sorted(range(router["experts"]), key=lambda e: (-float(z[t, e]), e))[:router["top"]]
        chosen.append(ids)
        weights.append(torch.softmax(torch.stack([z[t, e] for e in ids]), -1))
    return chosen, weights


def moe_ff(h, w, mlp):
    chosen, weights = route(h, w, mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in zip(chosen[t], weights[t]):
            out[t] += weight * gated_ff(h[t:t + 1], below(w, f"e{e}"))[0]
    if mlp.get("shared") is not None:
        shared = below(w, "shared")
        out = out + sigmoid(h @ shared["sg"].T) * gated_ff(h, shared)
    return out


# ------------------------------------------------------------------------------------ the model

MIXERS = {"latent_attention": latent_attention, "mlstm": mlstm, "mamba2": mamba2}


def below(w, prefix):
    return {k[len(prefix) + 1:]: v for k, v in w.items() if k.startswith(prefix + ".")}


def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, tensors, tokens, streams=None):
    """Logits [T, vocab] of one whole sequence; ``streams`` (a list) receives the residual
    stream after every layer."""
    w = {k: v.double() for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    tokens = [int(t) for t in tokens]
    x = w["embed"][tokens]
    bigram = (cfg.get("embedding") or {}).get("bigram")
    if bigram is not None:
        x = x + w["bigram"][bigram_rows(tokens, bigram)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}"
        y = MIXERS[layer["type"]](rms_norm(x, w[p + ".norm1"], eps), below(w, p + ".mix"),
                                  layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + moe_ff(rms_norm(x, w[p + ".norm2"], eps), below(w, p + ".mlp"), layer["mlp"])
        x = x + y
        if streams is not None:
            streams.append(x.clone())
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits
