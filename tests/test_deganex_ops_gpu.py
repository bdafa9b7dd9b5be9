"""Each mechanism of the Deganex architecture alone: the engine's kernel or part against the
plain function of tests/plain/deganex_plain.py, in 32-bit and (where rounding allows a sharp
bound) in bfloat16.  Inputs are made so that a fault shows: a query is built to meet ONE far
token's latent; decays run from slow enough that a lost state changes everything to strong enough
that a kept one does; a row's state is carried over portions of one and two tokens beside a
poisoned neighbour, and its slot is used again."""

import math

import pytest
import torch

from plain import deganex_plain as P
from test_titedra_ops_gpu import ctx
from test_vobosun_ops_gpu import DEV, bf16_exact, feed, i32, ops

pytestmark = pytest.mark.gpu


def rnd_of(seed):
    g = torch.Generator().manual_seed(seed)
    return g, lambda *shape, std=1.0: bf16_exact(torch.randn(shape, generator=g) * std)


def close(got, want, tol):
    """Root mean square of the difference over that of the wanted values, row by row."""
    err = (got.double() - want.double()).pow(2).mean(-1).sqrt() / want.double().pow(2).mean().sqrt()
    assert not torch.isnan(got).any()
    assert float(err.max()) < tol, (float(err.max()), int(err.argmax()))


# ------------------------------------------------------------------------------ norms of a sum

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d", [10, 33, 256, 1000])
def test_two_norms_of_a_stream_with_pending_terms_and_a_routed_sum(dtype, d):
    from scratch_llm_b200.parts.norm import RMSNorm
    from scratch_llm_b200.parts.stream import RoutedSum, Terms
    g, rnd = rnd_of(d)
    n, top, eps = 7, 3, 1e-3
    resid = rnd(n, d, std=2.0)
    terms = [(rnd(n, d), 1.0), (rnd(n, d), -0.75)]
    wa, wb = rnd(d, std=0.3) + 1.0, rnd(d, std=0.3) + 1.0
    place = torch.randperm(n * top, generator=g)
    place[4] = place[11] = -1                              # choices without a row of their own
    y, weights = rnd(n * top, d, std=1.5), torch.rand((n, top), generator=g)
    shared, gate = rnd(n, d), torch.randn((n, 9), generator=g)
    rows = y.double()[place.clamp(min=0)].view(n, top, d) * (place >= 0).view(n, top, 1)
    routed = (weights.double()[..., None] * rows).sum(1) \
        + torch.sigmoid(gate[:, 8:].double()) * shared.double()
    x = resid.double() + sum(c * t.double() for t, c in terms) + routed
    sum_ = Terms(tuple((t.to(DEV, dtype), c) for t, c in terms), RoutedSum(
        y.to(DEV), i32([[0] * top] * n), weights.to(DEV), i32(place.tolist()),
        shared.to(DEV, dtype), gate.to(DEV)[:, 8:]))
    torch.testing.assert_close(sum_.total().cpu(), (x - resid).float(), rtol=1e-5, atol=1e-5)
    a, b = RMSNorm(d, eps, ""), RMSNorm(d, eps, "")
    a.load({"": wa}, ctx(dtype))
    b.load({"": wb}, ctx(dtype))
    tol = dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)
    r = resid.clone().to(DEV)
    assert a.pairs_with(b) and not a.pairs_with(RMSNorm(d, 2 * eps, ""))
    ha, hb = a.forward_pair(r, sum_, b)
    torch.testing.assert_close(ha.float().cpu(), P.rms_norm(x, wa.double(), eps).float(), **tol)
    torch.testing.assert_close(hb.float().cpu(), P.rms_norm(x, wb.double(), eps).float(), **tol)
    torch.testing.assert_close(r.cpu(), x.float(), rtol=1e-5, atol=1e-5)     # the stream got the sum
    # only some rows, the stream untouched (the model's last norm)
    r2 = resid.clone().to(DEV)
    out = a.forward(r2, sum_, out_rows=i32([5, 0, 6]))
    torch.testing.assert_close(out.float().cpu(),
                               P.rms_norm(x, wa.double(), eps)[[5, 0, 6]].float(), **tol)
    assert torch.equal(r2.cpu(), resid)
    # nothing pending
    r3 = resid.clone().to(DEV)
    ha, hb = a.forward_pair(r3, None, b)
    torch.testing.assert_close(hb.float().cpu(), P.rms_norm(resid.double(), wb.double(),
                                                            eps).float(), **tol)
    assert torch.equal(r3.cpu(), resid)


# -------------------------------------------------------------------- the pair of two tokens

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("buckets, mul_prev, mul_cur", [(61, 7, 3), (1, 5, 5), (40, 0, 1),
                                                        (1009, 2_000_000_011, 3_000_000_019)])
def test_pairs_of_tokens_over_portions_and_used_slots(buckets, mul_prev, mul_cur, dtype):
    """The previous token is carried over portions of one and more tokens, two requests at a
    time, in a slot that an earlier request has left its own in; a token that the host has not
    read yet (pending) as the current one and, a step later, as the previous one."""
    from scratch_llm_b200.parts.token_pairs import HashedPairs
    g, rnd = rnd_of(buckets)
    vocab, d = 90, 24
    table, pairs = rnd(vocab, d), rnd(buckets + 1, d)
    part = HashedPairs(d, buckets, mul_prev, mul_cur)
    part.load({"": pairs}, ctx(dtype))
    emb = table.to(DEV, dtype)
    bigram = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}

    class Batch:
        pass

    state = i32([77, 77, 77])
    for first in (True, False):                      # the second time the slots are used again
        toks = {s: torch.randint(0, vocab, (17,), generator=g).tolist() for s in (2, 0)}
        fed = {2: 0, 0: 0}
        got = {2: [], 0: []}
        for cut in ([3, 1], [1, 2], [1, 1], [5, 1], [2, 9], [1, 1], [4, 2]):
            ids, pos, row, start = [], [], [], [0]
            pending = [0, 0]
            for r, (s, n) in enumerate(zip((2, 0), cut)):
                new = toks[s][fed[s]:fed[s] + n]
                if n == 1:                           # a token that only the device knows
                    pending[r] = new[0]
                    new = [-1 - r]
                ids += new
                pos += range(fed[s], fed[s] + n)
                row += [r] * n
                start.append(len(ids))
            b = Batch()
            ids, pos, row = ids + [0], pos + [0], row + [-1]          # a padding token
            b.token_ids, b.positions, b.token_row = i32(ids), i32(pos), i32(row)
            b.row_start, b.row_slot, b.pending_tokens = i32(start), i32([2, 0]), i32(pending)
            out = torch.empty((len(ids), d), dtype=torch.float32, device=DEV)
            part.embed(b, emb, out, 0.5, state)
            for r, s in enumerate((2, 0)):
                got[s].append(out[start[r]:start[r + 1]].cpu())
                fed[s] += cut[r]
        for s in (2, 0):
            rows = P.bigram_rows(toks[s], bigram)
            want = table[toks[s]] * 0.5 + pairs[rows]
            torch.testing.assert_close(torch.cat(got[s]), want, rtol=1e-6, atol=1e-6)
    assert state.tolist()[1] == 77                   # nobody's slot


# ------------------------------------------------------------------- gates of the recurrences

def test_state_space_gates():
    g, rnd = rnd_of(3)
    pre = torch.randn((50, 11), generator=g) * 4
    pre[3, 2], pre[4, 2] = 60.0, -60.0
    bias, a_log = rnd(5), rnd(5)
    la, w = (torch.empty((50, 5), device=DEV) for _ in range(2))
    ops().ssd_gates(pre.to(DEV)[:, 1:6], bias.to(DEV), a_log.to(DEV), la, w)
    dt = P.softplus(pre[:, 1:6].double() + bias.double())
    torch.testing.assert_close(w.cpu(), dt.float(), rtol=1e-5, atol=1e-30)
    torch.testing.assert_close(la.cpu(), (-torch.exp(a_log.double()) * dt).float(), rtol=1e-5,
                               atol=1e-30)


@pytest.mark.parametrize("cap", [2.0, 15.0, 40.0])
def test_matrix_memory_gates_keep_a_running_maximum(cap):
    """The maximum runs over rows of more than 256 tokens (the kernel's stride), over portions
    and single tokens, and starts at 0; a gate far above the others early on keeps it up."""
    g, rnd = rnd_of(int(cap))
    H, T = 3, 700
    pre = torch.randn((T, 2 * H), generator=g) * 6
    pre[:, H:] += 5.0                                  # forget gates near 1
    pre[:60, :H] -= 30.0                               # at first the start's 0 is the maximum
    pre[100, 0] = 200.0
    bi, bf = rnd(H), rnd(H)
    i = cap * torch.tanh((pre[:, :H].double() + bi.double()) / cap)
    f = -P.softplus(-(cap * torch.tanh((pre[:, H:].double() + bf.double()) / cap)))
    m, ms = torch.zeros(H, dtype=torch.float64), []
    for t in range(T):
        m = torch.maximum(f[t] + m, i[t])
        ms.append(m)
    ms = torch.stack(ms)
    before = torch.cat([torch.zeros(1, H, dtype=torch.float64), ms[:-1]])
    running = torch.zeros((4, H), device=DEV)
    running[1] = float("nan")
    t0 = 0
    for n in (1, 2, 300, 1, 31, 1, 260, 104):
        outs = [torch.full((n, H), float("nan"), device=DEV) for _ in range(3)]
        one = n == 1
        # a row without tokens beside it (its slot holds a NaN)
        ops().memory_gates(pre[t0:t0 + n].to(DEV), bi.to(DEV), bf.to(DEV), cap, running,
                           i32([0, 0, n]), i32([1, 2]), 2, *outs, one_each=one)
        s = slice(t0, t0 + n)
        tol = dict(rtol=1e-4, atol=2e-5)
        torch.testing.assert_close(outs[0].cpu(), (f + before - ms)[s].float(), **tol)
        torch.testing.assert_close(outs[1].cpu(), torch.exp(i - ms)[s].float(), **tol)
        torch.testing.assert_close(outs[2].cpu(), torch.exp(-ms)[s].float(), rtol=1e-4, atol=1e-30)
        assert float(outs[0].max()) <= 0.0 and float(outs[1].max()) <= 1.0
        t0 += n
    assert t0 == T
    torch.testing.assert_close(running[2].cpu(), ms[-1].float(), rtol=1e-5, atol=1e-5)


# ------------------------------------------------------------------------------------ the scan

SCANS = [  # heads, groups, key size, value size
    (4, 2, 16, 8), (3, 3, 6, 5), (2, 1, 48, 72), (4, 4, 64, 64), (2, 1, 128, 136), (1, 1, 9, 33),
    (2, 2, 200, 24), (2, 1, 256, 16), (1, 1, 300, 10), (1, 1, 1000, 4), (6, 2, 32, 40)]


def scan_case(H, G, N, V, T, seed, ones):
    g, rnd = rnd_of(seed)
    q, k, v = rnd(T, G, N), rnd(T, G, N, std=N ** -0.5), rnd(T, H, V)
    # decays from a few tokens' memory to one that hardly fades; one head forgets in a token
    rate = torch.tensor([[0.002, 0.3, 0.02, 1.0, 30.0, 0.08][h % 6] for h in range(H)])
    dt = torch.rand((T, H), generator=g) + 0.05
    dt[T // 2] = 0.0                                  # a token that writes and fades nothing
    skip = None if ones else rnd(H)
    y = P.ssd_scan(v.double(), k.double(), q.double(), dt.double(), rate.double(),
                   torch.zeros(H, dtype=torch.float64) if ones else skip.double())
    den = None
    if ones:
        den = P.ssd_scan(torch.ones((T, H, 1), dtype=torch.float64), k.double(), q.double(),
                         dt.double(), rate.double(), torch.zeros(H, dtype=torch.float64))[..., 0]
    return q, k, v, -rate[None] * dt, dt, skip, y, den


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("ones", [False, True])
@pytest.mark.parametrize("H, G, N, V", SCANS)
def test_scan_over_portions_and_slots(H, G, N, V, ones, chunked):
    """Two requests at a time through portions of all sizes (one and two tokens, chunk borders,
    several chunks), rows of one token beside long ones and a row without tokens; the slots
    held other numbers' worth of state before.  ``chunked``: the tensor-core kernels for every
    row of two tokens or more (where the sizes fit), else the token-by-token kernel."""
    dtype = torch.bfloat16 if chunked else torch.float32
    if chunked and (N % 16 or N > 256 or V % 8):
        pytest.skip("sizes the chunk kernels do not take")
    T = 333
    cases = {1: scan_case(H, G, N, V, T, 5, ones), 3: scan_case(H, G, N, V, T, 6, ones)}
    state = torch.full((5, H, V + ones, N), float("nan"), device=DEV)
    state[1], state[3] = 0.0, 0.0
    cuts = ([1, 2, 70, 1, 64, 128, 67], [200, 1, 2, 1, 64, 1, 64])
    fed = {1: 0, 3: 0}
    outs = {1: [], 3: []}
    dens = {1: [], 3: []}
    before = dict(ops().launch_counts)
    for a, b in zip(*cuts):
        rows = [(1, a), None, (3, b)]                 # the middle row brings nothing
        start = [0]
        pieces = {name: [] for name in "qkvlw"}
        for r in rows:
            n = 0
            if r is not None:
                s, n = r
                q, k, v, la, dt = cases[s][:5]
                sl = slice(fed[s], fed[s] + n)
                for name, t in zip("qkvlw", (q, k, v, la, dt)):
                    pieces[name].append(t[sl].reshape(n, -1))
            start.append(start[-1] + n)
        n = start[-1]
        # column slices of a wider buffer, as the projections' output is
        wide = torch.zeros((n, 2 * G * N + H * V + 64), dtype=dtype, device=DEV)
        c = [8 * -(-x // 8) for x in (G * N, 2 * (8 * -(-G * N // 8)))]
        wide = torch.zeros((n, c[1] + 8 * -(-H * V // 8)), dtype=dtype, device=DEV)
        views = wide[:, :G * N], wide[:, c[0]:c[0] + G * N], wide[:, c[1]:c[1] + H * V]
        for view, name in zip(views, "qkv"):
            view.copy_(torch.cat(pieces[name]).to(DEV, dtype))
        out = torch.full((n, H * V), float("nan"), device=DEV)
        den = torch.full((n, H), float("nan"), device=DEV) if ones else None
        skip = cases[1][5]
        # (both requests share the skip weights; see below)
        ops().gated_scan(*views, torch.cat(pieces["l"]).to(DEV), torch.cat(pieces["w"]).to(DEV),
                         state, i32(start), i32([1, 0, 3]), out, 3, G, N, V, longest=max(a, b),
                         ones_out=den, skip=None if ones else skip.to(DEV), scale=0.5,
                         min_chunked=2 if chunked else 0)
        for r, s in ((0, 1), (2, 3)):
            outs[s].append(out[start[r]:start[r + 1]].cpu())
            if ones:
                dens[s].append(den[start[r]:start[r + 1]].cpu())
            fed[s] += start[r + 1] - start[r]
    assert fed == {1: T, 3: T}
    used = ops().launch_counts.get("gated_scan_chunked", 0) - before.get("gated_scan_chunked", 0)
    assert used == (sum(max(c) >= 2 for c in zip(*cuts)) if chunked else 0)
    for s in (1, 3):
        _, _, v, _, _, skip, y, den = cases[s]
        if not ones:      # the plain rule's skip is not scaled
            y = 0.5 * (y - skip.double()[:, None] * v.double()) \
                + cases[1][5].double()[:, None] * v.double()
        else:
            y = 0.5 * y
        close(torch.cat(outs[s]), y.reshape(T, H * V), 2e-5)
        if ones:
            close(torch.cat(dens[s]), 0.5 * den, 2e-5)
    assert torch.isnan(state[[0, 2, 4]]).all()        # nobody else's state was touched


def test_scan_starts_from_what_the_slot_holds():
    H, G, N, V, T = 2, 1, 32, 16, 90
    q, k, v, la, dt, skip, y, _ = scan_case(H, G, N, V, T, 8, False)
    args = [t.reshape(T, -1).to(DEV, torch.bfloat16) for t in (q, k, v)]
    outs = []
    for start in (0.0, 1.0):
        for chunk in (0, 2):
            state = torch.full((1, H, V, N), start, device=DEV)
            out = torch.empty((T, H * V), device=DEV)
            ops().gated_scan(*args, la.to(DEV), dt.to(DEV), state, i32([0, T]), i32([0]), out, 1,
                             G, N, V, longest=T, skip=skip.to(DEV), min_chunked=chunk)
            outs.append((out.cpu(), state.cpu()))
    close(outs[0][0], y.reshape(T, -1), 2e-5)
    for a, b in ((0, 1), (2, 3)):
        close(outs[a][0], outs[b][0], 2e-5)
        close(outs[a][1].flatten(1), outs[b][1].flatten(1), 2e-5)
    assert (outs[2][0] - outs[0][0]).norm() > 0.5 * outs[0][0].norm()


# ---------------------------------------------------------------------------- around the scans

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps, C, extra", [(4, 24, 8), (3, 10, 5), (1, 16, 0), (2, 64, 24)])
def test_convolution_with_a_bias_over_portions(dtype, taps, C, extra):
    g, rnd = rnd_of(C)
    T = 40
    x, w, b = rnd(T, C), rnd(C, taps), rnd(C)
    want = P.silu(P.short_conv(x.double(), w.double(), b.double()))
    state = torch.zeros((2, max(1, taps - 1), C), dtype=dtype, device=DEV)
    state[0] = float("nan")
    got, t0 = [], 0
    wt = w.t().contiguous().to(DEV)
    for n in (1, 2, 9, 1, 1, 20, 6):
        buf = torch.zeros((n, C + extra), dtype=dtype, device=DEV)
        buf[:, :C] = x[t0:t0 + n].to(DEV, dtype)
        out = torch.empty((n, C), dtype=dtype, device=DEV)
        st = state if taps > 1 else None
        ops().conv_silu(buf, w.to(DEV), st, i32([0] * n), i32([0, n]), i32([1]), out, wt,
                        bias=b.to(DEV))
        ops().conv_state_update(buf, taps, st, i32([0, n]), i32([1]), 1)
        got.append(out.float().cpu())
        t0 += n
    torch.testing.assert_close(torch.cat(got), want.float(),
                               **(dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32
                                  else dict(rtol=1e-2, atol=1e-2)))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W, parts", [(24, 2), (30, 5), (256, 1), (4096, 4), (21, 7)])
def test_gate_ahead_of_a_norm_in_parts(W, parts, dtype):
    g, rnd = rnd_of(W + parts)
    n, eps = 6, 1e-4
    o = torch.randn((n, W), generator=g) * torch.logspace(-3, 1, W)      # parts of unequal size
    wide, gain = rnd(n, W + 16, std=2.0), rnd(W)
    out = torch.empty((n, W), dtype=dtype, device=DEV)
    ops().gate_part_norm(o.to(DEV), wide.to(DEV, dtype)[:, 8:8 + W], gain.to(DEV), eps, parts, out)
    want = P.grouped_norm(o.double() * P.silu(wide[:, 8:8 + W].double()), parts, gain.double(), eps)
    torch.testing.assert_close(out.float().cpu(), want.float(),
                               **(dict(rtol=2e-5, atol=1e-5) if dtype == torch.float32
                                  else dict(rtol=1e-2, atol=1e-2)))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_read_out_with_a_divisor_then_norm_and_gate(dtype):
    """eps is large beside some of the divided values: dividing before or after the norm is not
    the same."""
    g, rnd = rnd_of(7)
    n, H, V, eps = 9, 3, 20, 1e-3
    o = torch.randn((n, H * V), generator=g)
    den = torch.randn((n, H), generator=g) * 30
    floor = torch.rand((n, H), generator=g) * 20
    den[0, 0] = floor[0, 0] = 0.0                       # 1e-6 alone
    gate, gain = rnd(n, H * V), rnd(H * V)
    out = torch.empty((n, H * V), dtype=dtype, device=DEV)
    ops().head_norm_gate(o.to(DEV), gate.to(DEV, dtype), gain.to(DEV), eps, out, H,
                         gate_activation="sigmoid", divisor=(den.to(DEV), floor.to(DEV)))
    div = torch.maximum(den.abs(), floor).double() + 1e-6
    x = P.rms_unit(o.double().view(n, H, V) / div[..., None], eps).reshape(n, H * V)
    want = x * gain.double() * P.sigmoid(gate.double())
    torch.testing.assert_close(out.float().cpu(), want.float(),
                               **(dict(rtol=2e-5, atol=1e-5) if dtype == torch.float32
                                  else dict(rtol=1e-2, atol=1e-2)))


# ------------------------------------------------------------------------- the recurrent mixers

PORTIONS = [7, 2, 100, 1, 33, 2, 130, 3, 20, 2, 1, 1, 2, 1, 1]
OTHER = [3, 1, 40, 2, 1, 1, 9]


def feed_mixer(mixer, x, xb, dtype, position=None, page=8, portions=PORTIONS, other=OTHER):
    seen = []

    def run(batch, view, t0, t1, off):
        rows = torch.cat([xb[sum(seen):][:off], x[t0:t1]], 0) if off else x[t0:t1]
        seen.append(off)
        return mixer.forward(rows.to(DEV, dtype), batch, view, True, position)[off:].float().cpu()

    return feed([mixer.kv_spec()], [mixer.state_spec()], dtype, page, portions, run, other=other)


def recurrent_case(kind, m, width, seed):
    import deganex_util as U
    layer = {"mlstm": U.mlstm, "mamba2": U.mamba2}[kind](*m, mlp=None)
    cfg = U.config(20, width, [layer], bigram=None)
    w = {k[len("l0.mix."):]: v for k, v in U.random_tensors(cfg, seed).items()
         if k.startswith("l0.mix.")}
    return layer["mixer"], w


def make_recurrent(kind, m, width, w, eps, dtype):
    from scratch_llm_b200.parts.matrix_memory import MatrixMemory
    from scratch_llm_b200.parts.state_space import StateSpace
    mixer = MatrixMemory(width, m["heads"], m["dim"], m["vdim"], m["gate_cap"], eps) \
        if kind == "mlstm" else StateSpace(width, m["heads"], m["groups"], m["state"], m["vdim"],
                                           m["conv"], m["norm_groups"], eps)
    mixer.load(w, ctx(dtype))
    return mixer


RECURRENT = [("mlstm", (3, 6, 10, 4.0), 40), ("mlstm", (2, 48, 72, 12.0), 64),
             ("mlstm", (4, 32, 16, 30.0), 64), ("mlstm", (1, 9, 33, 8.0), 30),
             ("mamba2", (4, 10, 12, 2, 3, 5), 40), ("mamba2", (6, 24, 32, 1, 4, 1), 64),
             ("mamba2", (2, 64, 128, 2, 2, 4), 96), ("mamba2", (3, 7, 9, 3, 1, 3), 30)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind, sizes, width", RECURRENT)
@pytest.mark.parametrize("cut", ["whole", "decode", "portions"])
def test_recurrent_mixers(cut, kind, sizes, width, dtype):
    T, eps = sum(PORTIONS), 1e-5
    m, w = recurrent_case(kind, sizes, width, seed=width)
    g, rnd = rnd_of(1)
    x, xb = rnd(T, width), rnd(60, width)
    plain = P.mlstm if kind == "mlstm" else P.mamba2
    want = plain(x.double(), {k: v.double() for k, v in w.items()}, m, eps).float()
    mixer = make_recurrent(kind, m, width, w, eps, dtype)
    cuts = {"whole": ([T], None), "decode": ([T - 20] + [1] * 20, None),
            "portions": (PORTIONS, OTHER)}[cut]
    got = feed_mixer(mixer, x, xb, dtype, portions=cuts[0], other=cuts[1])
    if dtype == torch.float32:
        close(got, want, 1e-4)
    else:
        # (a head's divisor or root mean square may be small: single rows move by more)
        err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
        assert err.median() < 0.015 and err.max() < 0.08, (err.median(), err.max())


@pytest.mark.parametrize("kind, sizes, width", RECURRENT[1:2] + RECURRENT[5:6])
def test_a_recurrence_remembers_its_first_tokens(kind, sizes, width):
    """What a far token wrote still counts 300 tokens later, and is still the engine's: with
    slow decays the last outputs move when the first token is another one, by the same amount
    as the plain rule's."""
    T, eps = sum(PORTIONS), 1e-5
    m, w = recurrent_case(kind, sizes, width, seed=3)
    if kind == "mlstm":
        w["f.b"] = torch.full_like(w["f.b"], 11.0)
        w["f"] = torch.zeros_like(w["f"])
    else:
        w["A_log"] = torch.full_like(w["A_log"], -7.0)
    g, rnd = rnd_of(2)
    x, xb = rnd(T, width), rnd(60, width)
    x[0] *= 4.0
    x2 = x.clone()
    x2[0] = rnd(width, std=4.0)
    plain = P.mlstm if kind == "mlstm" else P.mamba2
    wd = {k: v.double() for k, v in w.items()}
    want, want2 = (plain(t.double(), wd, m, eps).float() for t in (x, x2))
    moved = (want - want2)[-1]
    assert moved.norm() > 3e-3 * want[-1].norm()
    mixer = make_recurrent(kind, m, width, w, eps, torch.float32)
    got, got2 = (feed_mixer(mixer, t, xb, torch.float32) for t in (x, x2))
    assert ((got - got2)[-1] - moved).norm() < 0.02 * moved.norm()


# ------------------------------------------------------------------------- latent attention

def seeking_case(H, d, r, dv, R, width, T, pairs, seed, base=5000.0, boost=8.0):
    """Weights and inputs of one latent attention in which token i of every pair (i, j) looks for
    token j.  The shared key part is not normed, so x_j times ``boost`` gives j a long one (its
    latent, and so its value, keeps its size); every head's rotated query rows are one matrix M,
    and x_i is solved so that M x_i is j's shared key part turned by the angle of j - i: after
    both are rotated by their positions they are parallel, and no other key can reach their
    score.  i's own latent has nothing to do with j's."""
    assert width >= r and r % 2 == 0
    g, rnd = rnd_of(seed)
    w = {"dkv": rnd(R + r, width, std=width ** -0.5), "dkv.norm": rnd(R, std=0.1) + 1.0,
         "uk": rnd(H * d, R, std=R ** -0.5), "uv": rnd(H * dv, R, std=R ** -0.5),
         "g": rnd(H * dv, width, std=2 * width ** -0.5),
         "o": rnd(width, H * dv, std=(H * dv) ** -0.5)}
    rows = rnd(r, width, std=width ** -0.5).double()                             # M
    x = rnd(T, width)
    assert not {i for i, _ in pairs} & {j for _, j in pairs}

    def turn(v, p):
        freq = torch.tensor([base ** (-2.0 * k / r) for k in range(r // 2)], dtype=torch.float64)
        c, s = torch.cos(p * freq), torch.sin(p * freq)
        out = torch.empty_like(v)
        out[0::2], out[1::2] = v[0::2] * c - v[1::2] * s, v[1::2] * c + v[0::2] * s
        return out

    for _, j in pairs:
        x[j] *= boost
    back = torch.linalg.pinv(rows)
    raw = []
    for i, j in pairs:
        key = w["dkv"].double()[R:] @ x[j].double()
        t = back @ turn(key, j - i)
        x[i] = bf16_exact((t / t.pow(2).mean().sqrt()).float())
        raw.append(float(turn(rows @ x[i].double(), i) @ turn(key, j)))
    scale = 30.0 / min(raw)                 # every sought key scores 30 or more, in every head
    q = torch.zeros((H, d + r, width), dtype=torch.float64)
    q[:, :d] = torch.randn((H, d, width), generator=g, dtype=torch.float64) \
        * 2.0 / (scale * math.sqrt(width * d))
    q[:, d:] = rows
    w["q"] = bf16_exact(q.reshape(H * (d + r), width).float())
    m = {"heads": H, "dim": d, "rot_dim": r, "vdim": dv, "kv_rank": R, "scale": scale,
         "rot": {"base": base, "dims": r}}
    return m, w, x


LATENT = [  # heads, dim, rot_dim, vdim, kv_rank, width, page
    (4, 16, 16, 24, 48, 64, 16),       # a cached vector of 64 entries
    (3, 8, 8, 10, 20, 48, 8),          # of 28, kept as 32
    (2, 20, 10, 12, 48, 72, 16),       # of 58, kept as 64; value columns off 16 bytes
    (16, 32, 32, 32, 96, 128, 16),     # of 128, many heads on one cached vector
    (20, 16, 16, 24, 48, 96, 16),      # of 64, more heads than one tile of queries holds
    (1, 8, 28, 1, 36, 40, 32),         # one head, one value channel (one gate per head)
    (2, 16, 32, 40, 256, 64, 64)]      # of 288: beyond the tensor-core kernels' sizes


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, d, r, dv, R, width, page", LATENT)
@pytest.mark.parametrize("cut", ["whole", "decode", "portions"])
def test_latent_attention_sees_far_keys_and_page_borders(cut, H, d, r, dv, R, width, page, dtype):
    """Queries near the end look for one token each: the first of the sequence, the second, a
    page's last place and the next page's first, one in the middle, and their own neighbour."""
    from scratch_llm_b200.parts.latent_attention import LatentAttention
    from scratch_llm_b200.parts.position import Rotary
    T, eps = 330, 1e-5
    pairs = [(T - 1, 1), (T - 2, page - 1), (T - 3, page), (T - 4, 5 * page + 1), (T - 5, 0),
             (T - 6, T - 7)]
    m, w, x = seeking_case(H, d, r, dv, R, width, T, pairs, seed=H * d + r)
    want = P.latent_attention(x.double(), {k: v.double() for k, v in w.items()}, m, eps).float()
    mixer = LatentAttention(width, H, d, r, dv, None, R, m["scale"], eps, gate="wide",
                            adjacent_pairs=r)
    assert "dq" not in mixer.param_specs() and mixer.param_specs()["g"].shape == (H * dv, width)
    mixer.load(w, ctx(dtype))
    pos = Rotary(r, m["rot"]["base"], 4096, interleaved=True, rot_dims=r)
    pos.load({}, ctx(dtype))
    portions = {"whole": [T], "decode": [T - 8] + [1] * 8,
                "portions": [7, 2, 100, 1, 33, 2, 152, 3, 20, 2, 1, 1, 2, 1, 1, 1, 1]}[cut]
    assert sum(portions) == T
    xb = bf16_exact(torch.randn((60, width), generator=torch.Generator().manual_seed(3)))
    got = feed_mixer(mixer, x, xb, dtype, pos, page, portions,
                     [3, 1, 40, 2, 1, 1, 9] if cut == "portions" else None)
    if dtype == torch.float32:
        torch.testing.assert_close(got, want, rtol=2e-4, atol=2e-4)
    else:
        # (scores of 30 carry bfloat16 errors of a tenth; the seekers have a margin, and 32-bit
        # above is sharp for every row)
        err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
        assert err.median() < 0.02 and err.max() < 0.3, (err.median(), err.max())
        assert err[[i for i, _ in pairs]].max() < 0.06


# ------------------------------------------------------------------------ routed feed-forward

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts, top, ff, shared", [(6, 2, 24, 40), (5, 1, 40, None), (3, 3, 16, 8),
                                                      (16, 4, 64, 64), (9, 5, 13, 7)])
def test_experts_weighted_by_a_softmax_over_the_chosen_and_a_gated_shared_one(experts, top, ff,
                                                                              shared, dtype):
    from scratch_llm_b200.parts.routed import RoutedExperts
    g, rnd = rnd_of(experts * 10 + top)
    width, n = 64, 90
    w = {"router": rnd(experts, width, std=2 * width ** -0.5)}
    names = {f"e{e}": ff for e in range(experts)}
    if shared:
        names["shared"] = shared
        w["shared.sg"] = rnd(1, width, std=2 * width ** -0.5)
    for name, f in names.items():
        w[f"{name}.gate"] = rnd(f, width, std=width ** -0.5)
        w[f"{name}.up"] = rnd(f, width, std=width ** -0.5)
        w[f"{name}.down"] = rnd(width, f, std=f ** -0.5)
    x = rnd(n, width)
    mlp = {"router": {"experts": experts, "top": top}, "shared": {"ff": shared} if shared else None}
    wd = {k: v.double() for k, v in w.items()}
    want = P.moe_ff(x.double(), wd, mlp).float()
    part = RoutedExperts(width, ff, experts, top, shared_size=shared, correction=False,
                         shared_gate=bool(shared))
    assert set(part.param_specs()) == set(w)
    part.load(w, ctx(dtype))
    xg = x.to(DEV, dtype)
    got = part.forward(xg).float().cpu()
    from scratch_llm_b200.parts.stream import Terms
    lazy = Terms.of(part.forward(xg, lazy=True)).total().cpu()
    few = part.forward(xg[40:45]).float().cpu()
    if dtype == torch.float32:
        torch.testing.assert_close(got, want, rtol=2e-4, atol=2e-4)
        torch.testing.assert_close(lazy, got, rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(few, got[40:45], rtol=1e-5, atol=1e-5)
        # the weights are the chosen logits' softmax
        chosen, weights = P.route(x.double(), wd, mlp["router"])
        logits = (x.double() @ wd["router"].T).float()
        buf = torch.zeros((n, experts + 3), device=DEV)
        buf[:, 2:2 + experts] = logits.to(DEV)
        ids, wts = ops().moe_route(buf[:, 2:2 + experts], None, None, experts, 1, 1, top)[:2]
        assert ids.cpu().tolist() == chosen
        torch.testing.assert_close(wts.cpu().double(), torch.stack(weights), rtol=1e-5, atol=1e-7)
    else:
        torch.testing.assert_close(lazy, got, rtol=2e-2, atol=2e-2)
        torch.testing.assert_close(few, got[40:45], rtol=2e-2, atol=2e-2)
        err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
        assert err.median() < 0.02 and err.quantile(0.9) < 0.05
