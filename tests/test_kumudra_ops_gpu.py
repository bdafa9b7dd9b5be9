"""Each mechanism of the Kumudra architecture alone: the engine's kernel or part against the plain
function of tests/plain/kumudra_plain.py, in 32-bit and (where rounding allows a sharp bound) in
bfloat16.  Inputs are made so that a fault shows: a query meets ONE key just inside or just outside
the window; decays run from none to ones that leave nothing within a token; a row's state is carried
over portions of one and two tokens beside a poisoned neighbour, and its slot is used again."""

import math

import pytest
import torch

import kumudra_util as U
from plain import kumudra_plain as P
from test_deganex_ops_gpu import OTHER, PORTIONS, close, feed_mixer, rnd_of
from test_titedra_ops_gpu import ctx
from test_vobosun_ops_gpu import DEV, bf16_exact, feed, i32, ops

pytestmark = pytest.mark.gpu


def doubles(w):
    return {k: v.double() for k, v in w.items()}


def tolerance(dtype, fine=1e-5, coarse=1e-2):
    return dict(rtol=fine, atol=fine) if dtype == torch.float32 else dict(rtol=coarse, atol=coarse)


# ---------------------------------------------------------------------------------- streams

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("S, d", [(1, 10), (2, 256), (3, 33), (4, 1000), (7, 48), (16, 20), (2, 12000)])
def test_streams_are_mixed_read_and_normed_in_one_pass(dtype, S, d):
    """Nothing pending, pending terms, a pending routed sum with choices that have no row; chosen
    rows only (nothing is written then); a layer norm with and without an offset, an RMS norm."""
    from scratch_llm_b200.parts.norm import LayerNorm, RMSNorm
    from scratch_llm_b200.parts.stream import RoutedSum, StreamUpdate, Terms
    g, rnd = rnd_of(S * d)
    n, top, eps = 7, 3, 1e-3
    parts = rnd(n, S, d, std=2.0)
    read, to, mix = rnd(S), rnd(S), rnd(S, S)
    terms = [(rnd(n, d), 0.8), (rnd(n, d), -0.75)]
    w, b = rnd(d, std=0.3) + 1.0, rnd(d)
    place = torch.randperm(n * top, generator=g)
    place[4] = place[11] = -1
    y, weights = rnd(n * top, d, std=1.5), torch.rand((n, top), generator=g)
    rows = y.double()[place.clamp(min=0)].view(n, top, d) * (place >= 0).view(n, top, 1)
    routed = (weights.double()[..., None] * rows).sum(1)
    out = sum(c * t.double() for t, c in terms)
    device_terms = tuple((t.to(DEV, dtype), c) for t, c in terms)
    device_routed = RoutedSum(y.to(DEV), i32([[0] * top] * n), weights.to(DEV), i32(place.tolist()),
                              None, None)
    cases = [(None, None), (Terms(device_terms), out), (Terms((), device_routed), routed),
             (Terms(device_terms, device_routed), out + routed)]
    norms = [LayerNorm(d, eps, "", bias=False), LayerNorm(d, eps, ""), RMSNorm(d, eps, "")]
    norms[0].load({"": w}, ctx(dtype))
    norms[1].load({"": w, "b": b}, ctx(dtype))
    norms[2].load({"": w}, ctx(dtype))
    plain = [lambda u: P.layer_norm(u, w.double(), eps),
             lambda u: P.layer_norm(u, w.double(), eps) + b.double(),
             lambda u: P.rms_unit(u, eps) * w.double()]
    old = parts.double().transpose(0, 1)
    for pending, value in cases:
        new = old if value is None else P.update_streams(old, value, mix.double(), to.double(), 1.0)
        update = None if value is None else StreamUpdate(pending, mix.to(DEV), to.to(DEV))
        for k in (range(3) if value is out else (0,)):
            for reading in (read, None):
                u = P.read_streams(new, torch.ones(S).double() if reading is None else read.double())
                want = plain[k](u).float()
                r = parts.clone().to(DEV)
                if update is not None:
                    torch.testing.assert_close(update.applied(r).cpu(),
                                               new.transpose(0, 1).float(), rtol=1e-4, atol=1e-4)
                given = None if reading is None else read.to(DEV)
                got = norms[k].forward(r, update, read=given)
                torch.testing.assert_close(got.float().cpu(), want, **tolerance(dtype, 3e-5))
                torch.testing.assert_close(r.cpu(), new.transpose(0, 1).float(), rtol=1e-5,
                                           atol=2e-5)
                r = parts.clone().to(DEV)
                few = norms[k].forward(r, update, out_rows=i32([5, 0, 5]), read=given)
                torch.testing.assert_close(few.float().cpu(), want[[5, 0, 5]],
                                           **tolerance(dtype, 3e-5))
                assert torch.equal(r.cpu(), parts)


def test_embedding_fills_every_part():
    g, rnd = rnd_of(4)
    table = rnd(11, 24)
    out = torch.empty((3, 5, 24), device=DEV)
    ops().embed(i32([4, 0, 10]), table.to(DEV), out, scale=0.25)
    want = (table[[4, 0, 10]] * 0.25)[:, None].expand(3, 5, 24)
    assert torch.equal(out.cpu(), want)


def test_layer_norm_without_an_offset():
    from scratch_llm_b200.parts.norm import LayerNorm
    g, rnd = rnd_of(9)
    for d in (24, 33):
        x, w, t = rnd(5, d), rnd(d), rnd(5, d)
        norm = LayerNorm(d, 1e-5, "", bias=False)
        norm.load({"": w}, ctx(torch.float32))
        got = norm.forward(x.clone().to(DEV), t.to(DEV))
        torch.testing.assert_close(got.cpu(), P.layer_norm((x + t).double(), w.double(),
                                                           1e-5).float(), rtol=1e-5, atol=1e-5)


# ------------------------------------------------------------------------------------ scans

CHANNEL_SCANS = [  # heads, key size, value size
    (4, 16, 8), (3, 6, 5), (2, 48, 72), (3, 64, 64), (2, 128, 136), (1, 9, 33), (2, 200, 24),
    (1, 256, 130), (1, 300, 10), (1, 1000, 4), (2, 31, 66)]


def channel_case(H, N, V, T, seed):
    g, rnd = rnd_of(seed)
    q, k, v = rnd(T, H, N), rnd(T, H, N, std=N ** -0.5), rnd(T, H, V)
    # channels that never fade, fade over hundreds of tokens, over a few, and within one
    rate = torch.tensor([0.0, 0.003, 0.1, 1.0, 20.0, 88.0])[torch.randint(0, 6, (H, N), generator=g)]
    log = -rate * (0.5 + torch.rand((T, H, N), generator=g)).clamp(max=1.0)
    log[T // 2] = 0.0                                 # a token that fades nothing
    log[T // 3] = -88.0                               # one that leaves nothing
    log[T // 3, :, ::3] = -0.01
    return q, k, v, log


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("bonus", [False, True])
@pytest.mark.parametrize("H, N, V", CHANNEL_SCANS)
def test_channel_scan_over_portions_and_slots(H, N, V, bonus, chunked, dtype):
    """Two requests at a time through portions of all sizes (one and two tokens, block and chunk
    borders, several chunks), rows of one token beside long ones and a row without tokens; slots of
    others hold NaN.  ``chunked``: the chunk kernels for every row of two tokens or more."""
    T = 333
    cases = {1: channel_case(H, N, V, T, 5), 3: channel_case(H, N, V, T, 6)}
    g, rnd = rnd_of(7)
    u = rnd(H, N) if bonus else None
    want = {}
    for s, (q, k, v, log) in cases.items():
        a = (q.double(), k.double(), v.double(), torch.exp(log.double()))
        want[s] = 0.5 * (P.bonus_scan(*a, u.double()) if bonus else P.decayed_scan(*a))
    state = torch.full((5, H, V, N), float("nan"), device=DEV)
    state[1], state[3] = 0.0, 0.0
    cuts = ([1, 2, 70, 1, 64, 128, 67], [200, 1, 2, 1, 64, 1, 64])
    fed, outs = {1: 0, 3: 0}, {1: [], 3: []}
    before = dict(ops().launch_counts)
    for a, b in zip(*cuts):
        start, pieces = [0], {name: [] for name in "qkvl"}
        for r in [(1, a), None, (3, b)]:              # the middle row brings nothing
            n = 0
            if r is not None:
                s, n = r
                for name, t in zip("qkvl", cases[s]):
                    pieces[name].append(t[fed[s]:fed[s] + n].reshape(n, -1))
            start.append(start[-1] + n)
        n = start[-1]
        # column slices of a wider buffer, as the projections' output is
        c = [8 * -(-x // 8) for x in (H * N, 2 * (8 * -(-H * N // 8)))]
        wide = torch.zeros((n, c[1] + 8 * -(-H * V // 8)), dtype=dtype, device=DEV)
        views = wide[:, :H * N], wide[:, c[0]:c[0] + H * N], wide[:, c[1]:c[1] + H * V]
        for view, name in zip(views, "qkv"):
            view.copy_(torch.cat(pieces[name]).to(DEV, dtype))
        out = torch.full((n, H * V), float("nan"), device=DEV)
        ops().channel_scan(*views, torch.cat(pieces["l"]).to(DEV), state, i32(start), i32([1, 0, 3]),
                           out, 3, H, N, V, longest=max(a, b),
                           bonus=None if u is None else u.to(DEV), scale=0.5,
                           min_chunked=2 if chunked else 0)
        for r, s in ((0, 1), (2, 3)):
            outs[s].append(out[start[r]:start[r + 1]].cpu())
            fed[s] += start[r + 1] - start[r]
    assert fed == {1: T, 3: T}
    name = "channel_scan_chunked"
    used = ops().launch_counts.get(name, 0) - before.get(name, 0)
    assert used == (sum(max(c) >= 2 for c in zip(*cuts)) if chunked else 0)
    for s in (1, 3):
        close(torch.cat(outs[s]), want[s].reshape(T, H * V), 2e-5)
    assert torch.isnan(state[[0, 2, 4]]).all()        # nobody else's state was touched


def test_channel_scan_starts_from_what_the_slot_holds():
    H, N, V, T = 2, 32, 16, 90
    q, k, v, log = channel_case(H, N, V, T, 8)
    log[T // 3] = -0.01
    args = [t.reshape(T, -1).to(DEV, torch.bfloat16) for t in (q, k, v)]
    outs = []
    for start in (0.0, 1.0):
        for chunk in (0, 2):
            state = torch.full((1, H, V, N), start, device=DEV)
            out = torch.empty((T, H * V), device=DEV)
            ops().channel_scan(*args, log.reshape(T, -1).to(DEV), state, i32([0, T]), i32([0]), out,
                               1, H, N, V, longest=T, min_chunked=chunk)
            outs.append((out.cpu(), state.cpu()))
    for a, b in ((0, 1), (2, 3)):
        close(outs[a][0], outs[b][0], 2e-5)
        close(outs[a][1].flatten(1), outs[b][1].flatten(1), 2e-5)
    assert (outs[2][0] - outs[0][0]).norm() > 0.5 * outs[0][0].norm()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, N, V", [(4, 16, 8), (3, 6, 5), (2, 48, 72), (3, 64, 64), (1, 300, 10)])
def test_scan_with_a_constant_decay_per_head_and_silu(H, N, V, dtype):
    """Decays that are one array for all tokens, no input weights, silu inside the token-by-token
    kernel or ahead of the chunk kernels."""
    T = 260
    g, rnd = rnd_of(N)
    q, k, v = rnd(T, H, N), rnd(T, H, N), rnd(T, H, V)
    decay = [[1.0, 0.9, 0.5, 0.01][h % 4] for h in range(H)]
    full = torch.tensor(decay, dtype=torch.float64)[None, :, None].expand(T, H, N)
    want = P.decayed_scan(P.silu(q.double()), P.silu(k.double()), P.silu(v.double()), full)
    log = torch.tensor([math.log(a) for a in decay], device=DEV)
    state = torch.zeros((2, H, V, N), device=DEV)
    state[0] = float("nan")
    got, t0 = [], 0
    for n in (1, 2, 30, 1, 150, 64, 12):
        proj = torch.cat([t[t0:t0 + n].reshape(n, -1) for t in (q, k, v)], 1).to(DEV, dtype)
        inside = n < 64
        if not inside:
            ops().silu_columns(proj)
        out = torch.empty((n, H * V), device=DEV)
        ops().gated_scan(proj[:, :H * N], proj[:, H * N:2 * H * N], proj[:, 2 * H * N:], log, None,
                         state, i32([0, n]), i32([1]), out, 1, H, N, V, longest=n, shortest=n,
                         silu=inside)
        got.append(out.cpu())
        t0 += n
    assert t0 == T
    close(torch.cat(got), want.reshape(T, -1), 2e-5 if dtype == torch.float32 else 1e-2)


# ---------------------------------------------------------------------------- around the scans

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d", [7, 30, 64, 520])
def test_token_shift_in_front_of_several_projections(d, dtype):
    g, rnd = rnd_of(d)
    T = 40
    h, mu, hb = rnd(T, d), rnd(5, d), rnd(30, d)
    prev = P.shifted(h)
    want = torch.stack([h + (prev - h) * mu[m] for m in range(5)])
    from scratch_llm_b200.parts import StateSpec
    portions, other = [1, 2, 9, 1, 1, 20, 4, 2], [5, 1, 2, 3]
    got, seen = [], []

    def run(batch, view, t0, t1, off):
        rows = torch.cat([hb[sum(seen):][:off], h[t0:t1]], 0).to(DEV, dtype)
        seen.append(off)
        out = torch.full((5, rows.shape[0], d), float("nan"), dtype=dtype, device=DEV)
        ops().shift_mix(rows, mu.to(DEV), view.state, batch.token_row, batch.row_start,
                        batch.row_slot, out)
        got.append(out[:, off:].float().cpu())
        return torch.zeros(1)

    feed([None], [StateSpec((d,), torch.float32)], dtype, 16, portions, run, other=other)
    torch.testing.assert_close(torch.cat(got, 1), want, **tolerance(dtype, 1e-6))


def test_token_shift_leaves_padding_alone():
    g, rnd = rnd_of(1)
    h, mu = rnd(6, 8), rnd(2, 8)
    state = torch.zeros((3, 8), device=DEV)
    out = torch.full((2, 6, 8), float("nan"), device=DEV)
    ops().shift_mix(h.to(DEV), mu.to(DEV), state, i32([0, 0, 1, -1, -1, -1]), i32([0, 2, 3, 3]),
                    i32([2, 1, 0]), out)
    assert torch.equal(state.cpu(), torch.stack([torch.zeros(8), h[2], h[1]]))
    assert torch.equal(out[:, 3:].cpu(), torch.zeros(2, 3, 8))
    assert not torch.isnan(out).any()


@pytest.mark.parametrize("n", [1, 19, 530])
@pytest.mark.parametrize("R, C", [(1, 5), (16, 96), (37, 300), (64, 1024), (130, 258)])
def test_log_decays_through_a_low_rank_pair(R, C, n):
    g, rnd = rnd_of(R)
    pre, w2t, bias = rnd(n, R + 3, std=2.0), rnd(R, C, std=R ** -0.5), rnd(C, std=6.0)
    bias[0], bias[1] = 200.0, -200.0                  # beyond both ends
    hidden = pre[:, 2:2 + R].double()
    for kind in ("sigmoid", "exp"):
        z = (torch.tanh(hidden) if kind == "exp" else hidden) @ w2t.double() + bias.double()
        want = P.log_sigmoid(z) / 3.0 if kind == "sigmoid" else -torch.exp(z)
        out = torch.empty((n, C), device=DEV)
        ops().lowrank_expand(pre.to(DEV), 2, w2t.to(DEV), out, bias=bias.to(DEV), log_decay=kind,
                             rate=1.0 / 3.0, tanh_in=kind == "exp")
        torch.testing.assert_close(out.cpu(), want.clamp(min=-88.0).float(), rtol=2e-5, atol=1e-6)
        assert float(out.max()) <= 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W, parts", [(24, 1), (30, 5), (2048, 1), (21, 7)])
def test_a_norm_and_then_a_gate(W, parts, dtype):
    g, rnd = rnd_of(W)
    n, eps = 5, 1e-3
    o, gate, gain = rnd(n, W, std=0.05), rnd(n, W + 3), rnd(W)
    for act in ("sigmoid", "silu"):
        f = P.sigmoid if act == "sigmoid" else P.silu
        x = P.rms_unit(o.double().view(n, parts, -1), eps).reshape(n, W) * gain.double()
        want = x * f(gate[:, 3:].double())
        out = torch.empty((n, W), dtype=dtype, device=DEV)
        ops().gate_part_norm(o.to(DEV), gate.to(DEV, dtype)[:, 3:], gain.to(DEV), eps, parts, out,
                             gate_activation=act, gate_after=True)
        torch.testing.assert_close(out.float().cpu(), want.float(), **tolerance(dtype, 2e-5))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("G, N, K", [(4, 42, 48), (4, 256, 1024), (3, 7, 20)])
def test_grouped_products_with_inputs_of_their_own(G, N, K, dtype):
    from scratch_llm_b200.parts.linear import GroupedLinear
    g, rnd = rnd_of(K)
    w = rnd(G, N, K, std=K ** -0.5)
    product = GroupedLinear(w.to(DEV, dtype))
    for m in (1, 3, 8, 9, 70):
        x = rnd(G, m, K)
        got = product(x.to(DEV, dtype))
        torch.testing.assert_close(got.float().cpu(), torch.einsum("gmk,gnk->gmn", x, w),
                                   **tolerance(dtype))


@pytest.mark.parametrize("experts, top", [(1, 1), (6, 2), (12, 4), (9, 9)])
def test_router_weights_are_scaled_and_uncorrected(experts, top):
    g, rnd = rnd_of(experts)
    n, d = 90, 24
    h, w = rnd(n, d), {"router": rnd(experts, d), "correction": rnd(experts, std=0.4)}
    ids, wts = P.route(h.double(), doubles(w), {"experts": experts, "top": top, "scale": 1.7})
    z = (h @ w["router"].T).to(DEV)
    for rows in (n, 3):                               # the general kernels, and the one for few tokens
        got_ids, got = ops().moe_route(z[:rows], w["correction"].to(DEV), None, experts, 1, 1, top,
                                       flags=ops().MOE_SIGMOID, scale=1.7)[:2]
        assert got_ids.cpu().tolist() == ids[:rows]
        torch.testing.assert_close(got.cpu(), torch.tensor(wts[:rows]).float(), rtol=1e-5, atol=1e-6)


# -------------------------------------------------------------------------------- attention

ATTENTION = [  # heads, kv heads, dim, vdim, rot dims, window, page, scaling
    (8, 2, 64, 48, 32, 40, 16, None), (4, 2, 16, 24, 8, 13, 8, (4.0, 1.0, 3.0, 60)),
    (3, 3, 20, 12, 6, 16, 16, None), (2, 1, 128, 128, 128, 65, 32, (8.0, 1.0, 4.0, 400)),
    (4, 1, 64, 64, 16, 128, 64, (2.0, 0.5, 0.5, 100)), (2, 2, 12, 30, 2, 1, 16, None),
    (6, 3, 32, 64, 32, 500, 16, None), (4, 2, 64, 64, 6, 40, 16, (3.0, 1.0, 2.0, 80)),
    (2, 2, 60, 64, 22, 33, 16, None), (4, 2, 120, 128, 40, 90, 64, None)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, G, D, Dv, rot, window, page, scaled", ATTENTION)
@pytest.mark.parametrize("cut", ["whole", "decode", "portions"])
def test_attention_at_the_window_s_edges(cut, H, G, D, Dv, rot, window, page, scaled, dtype):
    """Queries, in the prompt and among the last tokens, are copies of the tokens window - 1 before
    them (the farthest that is seen) and window before them (not seen any more), of page borders
    and of themselves; their scores stand out by far."""
    g, rnd = rnd_of(H * D + window)
    width, T = 40, 330
    m = U.left(H, G, D, Dv, window, rot, base=5000.0,
               scaled=None if scaled is None else U.scaling(*scaled))
    w = {"q": rnd(H * D, width, std=width ** -0.5), "v": rnd(G * Dv, width, std=width ** -0.5),
         "o": rnd(width, H * Dv, std=(H * Dv) ** -0.5), "q.b": rnd(H * D, std=0.2),
         "k.b": rnd(G * D, std=0.2), "v.b": rnd(G * Dv, std=0.2)}
    # each kv head's key matrix is its first query head's: a token meets its own copy strongly
    w["k"] = torch.cat([w["q"][(h * (H // G)) * D:(h * (H // G) + 1) * D] for h in range(G)], 0)
    x = rnd(T, width)
    looking = [T - 1, T - 2, T - 5, 200, 201, 215]
    for n, i in enumerate(looking):
        back = window - 1 if n % 2 == 0 else window
        if 0 < back <= i and i - back not in looking:
            x[i] = x[i - back] = rnd(width, std=3.0)
    for i, j in ((T - 7, 5 * page), (T - 8, 5 * page - 1)):
        if i - j < window:
            x[i] = x[j] = rnd(width, std=3.0)
    want = P.window_attention(x.double(), doubles(w), m).float()
    if window > 1:          # one token more or less in the window shows
        for size in (window - 1, window + 1):
            other = P.window_attention(x.double(), doubles(w), {**m, "mask": {"size": size}})
            if window < T:
                assert (other.float() - want).abs().max() > 0.05 * want.abs().max()
    from scratch_llm_b200.parts.attention import GQAttention
    from scratch_llm_b200.parts.position import Rotary
    mixer = GQAttention(width, H, G, D, m["scale"], window, names={n: n for n in "qkvo"},
                        value_dim=Dv, bias=True)
    mixer.load(w, ctx(dtype))
    pos = Rotary(D, 5000.0, 4096, interleaved=False, rot_dims=rot, llama3=m["rot"]["scaling"])
    pos.load({}, ctx(dtype))
    portions = {"whole": [T], "decode": [T - 10] + [1] * 10,
                "portions": [7, 2, 100, 1, 33, 2, 152, 3, 18, 2, 1, 1, 2, 1, 1, 1, 1, 1, 1]}[cut]
    assert sum(portions) == T
    got = feed_mixer(mixer, x, rnd(60, width), dtype, pos, page, portions, None)
    if dtype == torch.float32:
        torch.testing.assert_close(got, want, rtol=2e-4, atol=2e-4)
    else:
        err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
        assert err.max() < 0.06, (err.max(), err.argmax())


# ------------------------------------------------------------------------- the recurrent mixers

def mixer_case(kind, sizes, width, seed):
    layer = {"gla": U.gla, "lightning": U.lightning,
             "time_mixing": lambda h, d: U.parallel(U.left(1, 1, 4, 4, 5, 2), h, d)}[kind](*sizes)
    cfg = U.config(20, width, [layer])
    prefix = "l0.mix.right." if kind == "time_mixing" else "l0.mix."
    w = {k[len(prefix):]: v for k, v in U.random_tensors(cfg, seed).items() if k.startswith(prefix)}
    m = layer["mixer"]["right"] if kind == "time_mixing" else layer["mixer"]
    return m, w, {"gla": P.gla, "lightning": P.lightning, "time_mixing": P.time_mixing}[kind]


def make_mixer(kind, m, width, w, eps, dtype):
    from scratch_llm_b200.parts.linear_attention import GatedLinearAttention, LightningAttention
    from scratch_llm_b200.parts.time_mixing import TimeMixing
    if kind == "time_mixing":
        mixer = TimeMixing(width, m["heads"], m["dim"], eps)
    elif kind == "gla":
        mixer = GatedLinearAttention(width, m["heads"], m["dim"], m["vdim"], m["tau"], eps)
    else:
        mixer = LightningAttention(width, m["heads"], m["dim"], m["vdim"], m["decay"], eps)
    mixer.load(w, ctx(dtype))
    return mixer


RECURRENT = [("gla", (3, 10, 6, 4.0), 40), ("gla", (2, 80, 72, 12.0), 64), ("gla", (1, 9, 33, 1.0), 30),
             ("gla", (4, 64, 64, 16.0), 128),
             ("lightning", (3, 10, 6, [0.0, 0.5, 1.0]), 40), ("lightning", (2, 48, 72, [0.3, 0.99]), 64),
             ("lightning", (1, 9, 33, [0.9]), 30), ("lightning", (2, 64, 64, [0.95, 0.999]), 128),
             ("time_mixing", (3, 10), 40), ("time_mixing", (2, 48), 64), ("time_mixing", (1, 33), 30),
             ("time_mixing", (4, 64), 128)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind, sizes, width", RECURRENT)
@pytest.mark.parametrize("cut", ["whole", "decode", "portions"])
def test_recurrent_mixers(cut, kind, sizes, width, dtype):
    T, eps = sum(PORTIONS), 1e-5
    m, w, plain = mixer_case(kind, sizes, width, seed=width)
    g, rnd = rnd_of(1)
    x, xb = rnd(T, width), rnd(60, width)
    want = plain(x.double(), doubles(w), m, eps).float()
    mixer = make_mixer(kind, m, width, w, eps, dtype)
    cuts = {"whole": ([T], None), "decode": ([T - 20] + [1] * 20, None),
            "portions": (PORTIONS, OTHER)}[cut]
    got = feed_mixer(mixer, x, xb, dtype, portions=cuts[0], other=cuts[1])
    if dtype == torch.float32:
        close(got, want, 1e-4)
    else:
        # (a head's root mean square may be small: single rows move by more)
        err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
        assert err.median() < 0.015 and err.max() < 0.1, (err.median(), err.max())


@pytest.mark.parametrize("kind, sizes, width", [("gla", (2, 48, 32, 8.0), 64),
                                                ("lightning", (2, 48, 32, [1.0, 1.0]), 64),
                                                ("time_mixing", (2, 32), 64)])
def test_a_recurrence_remembers_its_first_tokens(kind, sizes, width):
    """What a far token wrote still counts 300 tokens later, by the plain rule's amount."""
    T, eps = sum(PORTIONS), 1e-5
    m, w, plain = mixer_case(kind, sizes, width, seed=3)
    if kind == "gla":
        w["a2.b"] = torch.full_like(w["a2.b"], 9.0)
        w["a2"] = torch.zeros_like(w["a2"])
    elif kind == "time_mixing":
        w["w0"] = torch.full_like(w["w0"], -9.0)
        w["w2"] = torch.zeros_like(w["w2"])
    g, rnd = rnd_of(2)
    x, xb = rnd(T, width), rnd(60, width)
    x[0] *= 4.0
    x2 = x.clone()
    x2[0] = rnd(width, std=4.0)
    want, want2 = (plain(t.double(), doubles(w), m, eps).float() for t in (x, x2))
    moved = (want - want2)[-1]
    assert moved.norm() > 3e-3 * want[-1].norm()
    mixer = make_mixer(kind, m, width, w, eps, torch.float32)
    got, got2 = (feed_mixer(mixer, t, xb, torch.float32) for t in (x, x2))
    assert ((got - got2)[-1] - moved).norm() < 0.02 * moved.norm()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("scales", [(1.0, 1.0), (0.6, -1.3), (0.0, 0.7), (0.7, 0.0), (0.0, 0.0)])
def test_two_mixers_share_one_output_product(scales, dtype):
    """Attention and time mixing side by side through one output matrix (or two, where the side that
    cannot scale its activations has the weight 0), over portions beside a neighbour."""
    from scratch_llm_b200.parts.position import Rotary
    from scratch_llm_b200.parts.side_by_side import SideBySide
    width, T, eps = 48, sum(PORTIONS), 1e-5
    layer = U.parallel(U.left(4, 2, 12, 20, 30, 8), 3, 14, *scales)
    w = {k[len("l0.mix."):]: v for k, v in
         U.random_tensors(U.config(20, width, [layer]), 5).items() if k.startswith("l0.mix.")}
    g, rnd = rnd_of(3)
    x, xb = rnd(T, width), rnd(60, width)
    want = P.parallel(x.double(), doubles(w), layer["mixer"], eps).float()
    mixer = SideBySide(
        {"kind": "gqa_attention", "args": dict(
            hidden_size=width, n_heads=4, n_kv_heads=2, head_dim=12, value_dim=20, scale=12 ** -0.5,
            bias=True, window=30, names={n: n for n in "qkvo"})},
        {"kind": "time_mixing", "args": dict(hidden_size=width, n_heads=3, head_dim=14, eps=eps)},
        *scales)
    mixer.load(w, ctx(dtype))
    pos = Rotary(12, 10000.0, 512, interleaved=False, rot_dims=8)
    pos.load({}, ctx(dtype))

    class Total:        # the sum of the terms
        kv_spec, state_spec = mixer.kv_spec, mixer.state_spec

        @staticmethod
        def forward(*args):
            return mixer.forward(*args).total()

    got = feed_mixer(Total, x, xb, dtype, pos)
    assert (mixer._joint is not False) == (scales[0] != 0.0 or scales[1] == 0.0)
    if not any(scales):
        assert float(got.abs().max()) == 0.0
        return
    close(got, want, 1e-4 if dtype == torch.float32 else 0.1)
