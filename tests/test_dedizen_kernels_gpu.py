"""The kernels and part options that Dedizen added, each against the plain function of the same mechanism (float64 on the
CPU), on sizes the tiny models do not reach, cut into portions and decoded, over hand-made paged caches and state slots,
with inputs made so that a fault shows: a write read back after hundreds of tokens, a key that stands out just inside and
just outside a chunk, gates at both ends, slots that are used again."""

import pytest
import torch

import plain_dedizen as pd

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def F():
    from mini_infer_b200.ops import functional
    return functional


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def close(got, want, tol):
    return float((got.double().cpu() - want).abs().max()) <= tol * max(float(want.abs().max()), 1e-30)


def bf(x):
    return x.to(torch.bfloat16).float()


# --------------------------------------------------------------------------- #
# matrix memories
# --------------------------------------------------------------------------- #

def memory_case(H, d, dv, lens, seed, log_gates, pad=3):
    """Projections ``[T, q | k | v | output gate | i | f]`` of several requests, rounded to bfloat16 so that every form of
    the kernels reads the same numbers, and the plain read-outs (before norm and gate, and after)."""
    g = torch.Generator().manual_seed(seed)
    n_qk, n_v = H * d, H * dv
    cols = (pad, pad + n_qk, pad + 2 * n_qk)
    col_g = pad + 2 * n_qk + n_v
    width = col_g + n_v + 2 * H
    if pad % 8 == 0:
        width = -(-width // 8) * 8                        # rows, and with them heads of whole eights, on 16-byte boundaries
    xs = [bf(torch.randn(n, width, generator=g)) for n in lens]
    for x in xs:
        x[:, col_g + n_v:] *= 2.0
    extra = dict(bi=torch.randn(H, generator=g), bf=2 + torch.randn(H, generator=g), cap=5.0,
                 decay=torch.tensor([[0.5, 0.9, 0.99, 1.0, 0.05][h % 5] for h in range(H)]),
                 w=1 + 0.2 * torch.randn(n_v, generator=g), cols=cols, col_g=col_g, col_i=col_g + n_v, eps=1e-5)
    want = []
    for x in xs:
        z, T = x.double(), x.shape[0]
        q, k = z[:, cols[0]:cols[0] + n_qk].reshape(T, H, d), z[:, cols[1]:cols[1] + n_qk].reshape(T, H, d)
        v = z[:, cols[2]:cols[2] + n_v].reshape(T, H, dv)
        if log_gates:
            c = extra["cap"]
            i = c * torch.tanh((z[:, extra["col_i"]:extra["col_i"] + H] + extra["bi"].double()) / c)
            f = pd.log_sigmoid(c * torch.tanh((z[:, extra["col_i"] + H:extra["col_i"] + 2 * H] + extra["bf"].double()) / c))
            o = pd.matrix_memory(q * d ** -0.5, k, v, i, f)
            y = pd.unit_rms(o, 1e-5).reshape(T, n_v) * extra["w"].double() * pd.sigmoid(z[:, col_g:col_g + n_v])
        else:
            o = pd.fixed_decay_memory(pd.silu(q), pd.silu(k), pd.silu(v), extra["decay"].double())
            y = o.reshape(T, n_v)
        want.append(y)
    return xs, want, extra


def run_memory(H, d, dv, xs, extra, cuts, log_gates, chunks, dtype, slots=None, decode=True):
    """Every request fed in portions ``cuts[r]``, side by side; steps of one token per request take the decode kernel
    (in bfloat16), the others the walk or, with ``chunks``, the chunks.  Slots are dirty before and zeroed at the start."""
    fn = F()
    st = fn.MemoryState(H, d, dv, log_gates)
    slots = slots or list(range(len(xs)))
    state = torch.randn(max(slots) + 2, st.floats + 4, generator=torch.Generator().manual_seed(1)).to(DEV)
    untouched = [s for s in range(state.shape[0]) if s not in slots]
    before = state[untouched].clone()
    state[slots] = 0.0
    gates = fn.LogGates(extra["col_i"], extra["col_i"] + H, extra["bi"].to(DEV), extra["bf"].to(DEV), extra["cap"]) if log_gates else None
    decay = None if log_gates else extra["decay"].to(DEV)
    fed, got = [0] * len(xs), [[] for _ in xs]
    kw = dict(gates=gates, decay=decay, q_scale=d ** -0.5 if log_gates else 1.0, silu=not log_gates)
    for step in range(max(len(c) for c in cuts)):
        live = [r for r in range(len(xs)) if step < len(cuts[r])]
        rows = [xs[r][fed[r]:fed[r] + cuts[r][step]] for r in live]
        proj = torch.cat(rows).to(DEV).contiguous()
        starts = [sum(r.shape[0] for r in rows[:n]) for n in range(len(rows) + 1)]
        args = (proj, extra["cols"], st, state, i32(starts), i32([slots[r] for r in live]))
        longest = max(cuts[r][step] for r in live)
        if decode and longest == 1:
            y = fn.memory_decode(*args, gate_col=extra["col_g"], weight=extra["w"].to(DEV), eps=1e-5, out_dtype=dtype, **kw)
        else:
            rows = proj
            if chunks:
                rows = proj.to(torch.bfloat16)
                y = fn.memory_chunks(rows, *args[1:], longest, gate_rows=proj, **kw)
            else:
                y = fn.memory_scan(*args, **kw)
            if log_gates:
                o, den, gv = y
                y = fn.memory_finish(o, rows, extra["col_g"], extra["w"].to(DEV), 1e-5, dtype, H, den, gv)
        for n, r in enumerate(live):
            got[r].append(y[starts[n]:starts[n + 1]].float().cpu())
            fed[r] += cuts[r][step]
    assert torch.equal(state[untouched], before)           # a slot of no request is left alone
    return [torch.cat(g) for g in got]


SIZES = [(1, 1, 1), (3, 10, 14), (2, 33, 17), (4, 64, 128), (2, 130, 70), (1, 256, 300), (5, 16, 64)]


@pytest.mark.parametrize("H,d,dv", SIZES)
@pytest.mark.parametrize("log_gates", [True, False])
def test_memory_walked_in_any_cut(H, d, dv, log_gates):
    lens = [90, 1, 37]
    xs, want, extra = memory_case(H, d, dv, lens, H + d + dv, log_gates)
    runs = []
    for cuts in ([[90], [1], [37]], [[40] + [1] * 50, [1], [2, 3, 5, 7, 20]], [[2] * 45, [1], [36, 1]]):
        got = run_memory(H, d, dv, xs, extra, cuts, log_gates, False, torch.float32, slots=[4, 0, 2], decode=False)
        runs.append(got)
        for r in range(3):
            # a one-number head is its own sign after the norm; elsewhere rounding is all there is
            assert close(got[r], want[r], 2e-4 if log_gates else 3e-6), (cuts, r)
    for other in runs[1:]:
        assert all(torch.equal(a, b) for a, b in zip(other, runs[0]))        # the same bits however it was cut


@pytest.mark.parametrize("H,d,dv", SIZES)
@pytest.mark.parametrize("log_gates", [True, False])
@pytest.mark.parametrize("pad", [3, 8])
def test_memory_in_chunks_and_decoded(H, d, dv, log_gates, pad):
    """Long portions over chunks of 64 tokens, portions that end inside a chunk, single tokens on the decode kernel.  The
    projections are bfloat16 numbers already, so the forms differ from the plain sums by what float and a pair of bfloat16
    lose only (silu, whose result the chunks round to bfloat16, aside)."""
    lens = [300, 1, 70, 65]
    xs, want, extra = memory_case(H, d, dv, lens, 7 * H + d + dv, log_gates, pad)
    tol = 1e-3 if log_gates else 8e-3
    for cuts in ([[300], [1], [70], [65]], [[129, 64, 63] + [1] * 44, [1], [64, 6], [2, 63]],
                 [[250] + [1] * 50, [1], [20] + [1] * 50, [15] + [1] * 50]):
        got = run_memory(H, d, dv, xs, extra, cuts, log_gates, True, torch.float32, slots=[1, 5, 0, 3])
        for r in range(4):
            assert close(got[r], want[r], tol), (cuts, r)


def test_decode_rounds_to_bfloat16_on_the_way_out():
    xs, want, extra = memory_case(3, 32, 40, [12], 3, True)
    got = run_memory(3, 32, 40, xs, extra, [[1] * 12], True, True, torch.bfloat16)
    assert close(got[0], want[0], 8e-3)


@pytest.mark.parametrize("log_gates", [True, False])
def test_a_write_is_read_back_after_hundreds_of_tokens(log_gates):
    """One token's key and value stand out; every later key is orthogonal to it and the last query asks for it."""
    H, d, dv, T = 2, 32, 48, 420
    g = torch.Generator().manual_seed(4)
    xs, _, extra = memory_case(H, d, dv, [T], 4, log_gates, pad=0)
    x = xs[0]
    c = extra["cols"]
    for h in range(H):
        x[:, c[1] + h * d] = 0.0 if log_gates else -30.0          # (silu of -30 is nothing)
        x[5, c[1] + h * d:c[1] + (h + 1) * d] = -30.0 if not log_gates else 0.0
        x[5, c[1] + h * d] = 8.0
        x[T - 1, c[0] + h * d:c[0] + (h + 1) * d] = 0.0 if log_gates else -30.0
        x[T - 1, c[0] + h * d] = 4.0
    x[5, c[2]:c[2] + H * dv] = bf(torch.randn(H * dv, generator=g) * 3)
    if log_gates:
        x[:, extra["col_i"]:extra["col_i"] + H] = -2.0
        x[5, extra["col_i"]:extra["col_i"] + H] = 4.0
        x[:, extra["col_i"] + H:extra["col_i"] + 2 * H] = 8.0                             # forget gates near one
        i = extra["cap"] * torch.tanh((x[:, extra["col_i"]:extra["col_i"] + H].double() + extra["bi"].double()) / extra["cap"])
        f = pd.log_sigmoid(extra["cap"] * torch.tanh((x[:, extra["col_i"] + H:extra["col_i"] + 2 * H].double() + extra["bf"].double()) / extra["cap"]))
        z = x.double()
        o = pd.matrix_memory(z[:, c[0]:c[0] + H * d].reshape(T, H, d) * d ** -0.5, z[:, c[1]:c[1] + H * d].reshape(T, H, d),
                             z[:, c[2]:c[2] + H * dv].reshape(T, H, dv), i, f)
        want = pd.unit_rms(o, 1e-5).reshape(T, H * dv) * extra["w"].double() * pd.sigmoid(z[:, extra["col_g"]:extra["col_g"] + H * dv])
    else:
        extra["decay"] = torch.tensor([1.0, 0.999])
        z = pd.silu(x.double())
        want = pd.fixed_decay_memory(*(z[:, a:a + H * n].reshape(T, H, n) for a, n in zip(c, (d, d, dv))),
                                     extra["decay"].double()).reshape(T, H * dv)
        assert float(want[T - 1].abs().max()) > 10                            # the far value is what is read
    for cuts, chunks in (([T], False), ([T], True), ([300] + [1] * 120, True), ([3, 61, 130, 1, 225], True), ([2] * 210, False)):
        got = run_memory(H, d, dv, [x], extra, [cuts], log_gates, chunks, torch.float32)[0]
        assert close(got[T - 1], want[T - 1], 1e-2 if chunks and not log_gates else 1e-4), (cuts, chunks)
        assert close(got, want, 1e-2 if chunks and not log_gates else 3e-4), (cuts, chunks)


def test_gates_at_both_ends():
    """Input gates at their caps, forget gates near 0 and near 1, in stretches: the running maximum jumps up, stays, and
    falls far; chunks whose decays sum to hundreds keep the weights of neighbours exact."""
    H, d, dv, T = 3, 16, 24, 260
    xs, _, extra = memory_case(H, d, dv, [T], 8, True, pad=0)
    x, c, ci = xs[0], extra["cols"], extra["col_i"]
    extra["cap"] = 15.0
    g = torch.Generator().manual_seed(9)
    x[:, ci:ci + H] = bf(torch.randn(T, H, generator=g) * 20)
    x[:, ci + H:ci + 2 * H] = bf(torch.randn(T, H, generator=g) * 20)
    x[100:180, ci + H:ci + 2 * H] = -60.0                                     # forget everything at every token
    x[180:, ci:ci + H] = -60.0                                      # and write next to nothing
    z = x.double()
    i = 15 * torch.tanh((z[:, ci:ci + H] + extra["bi"].double()) / 15)
    f = pd.log_sigmoid(15 * torch.tanh((z[:, ci + H:ci + 2 * H] + extra["bf"].double()) / 15))
    o = pd.matrix_memory(z[:, c[0]:c[0] + H * d].reshape(T, H, d) * d ** -0.5, z[:, c[1]:c[1] + H * d].reshape(T, H, d),
                         z[:, c[2]:c[2] + H * dv].reshape(T, H, dv), i, f)
    want = pd.unit_rms(o, 1e-5).reshape(T, H * dv) * extra["w"].double() * pd.sigmoid(z[:, extra["col_g"]:extra["col_g"] + H * dv])
    for cuts, chunks in (([T], False), ([T], True), ([130] + [1] * 130, True)):
        got = run_memory(H, d, dv, [x], extra, [cuts], True, chunks, torch.float32)[0]
        assert bool(torch.isfinite(got).all())
        err = (got.double() - want).abs().max(dim=1).values / want.abs().max()
        assert float(err.max()) <= 2e-3 and float(err.median()) <= 2e-5, (cuts, chunks, float(err.max()))


# --------------------------------------------------------------------------- #
# the gated linear recurrence per channel
# --------------------------------------------------------------------------- #

def lru_case(W, blocks, taps, lens, seed):
    g = torch.Generator().manual_seed(seed)
    n = W // blocks
    r = lambda *s, std=1.0: torch.randn(*s, generator=g) * std
    p = {"conv": r(W, taps, std=0.6), "conv.b": r(W, std=0.3), "x.b": r(W, std=0.5), "y.b": r(W, std=0.5),
         "ra": bf(r(blocks, n, n, std=1.5 * n ** -0.5)), "ri": bf(r(blocks, n, n, std=1.5 * n ** -0.5)),
         "ra.b": r(W, std=0.7), "ri.b": r(W, std=0.7), "lam": r(W, std=2.0) - 3.0}
    xs = [r(k, 2 * W + 5) for k in lens]                     # y from column 2 on, x from column W + 3 on
    want, us = [], []
    for x in xs:
        z, P = x.double(), {k: v.double() for k, v in p.items()}
        u = pd.causal_conv(z[:, W + 3:2 * W + 3] + P["x.b"], P["conv"], P["conv.b"])
        rr = pd.sigmoid(pd.block_product(u, P["ra"], P["ra.b"].reshape(blocks, n)))
        ii = pd.sigmoid(pd.block_product(u, P["ri"], P["ri.b"].reshape(blocks, n)))
        us.append((u, rr, ii))
        want.append(pd.real_gated_lru(u, rr, ii, P["lam"]) * pd.gelu_tanh(z[:, 2:W + 2] + P["y.b"]))
    return p, xs, us, want


def run_lru(W, blocks, taps, p, xs, cuts, dtype, segments, slots, decode=True, out_dtype=torch.float32):
    fn = F()
    d = {k: v.to(DEV) for k, v in p.items()}
    d["rate"] = (-8 * pd.softplus(p["lam"].double())).float().to(DEV)
    wr, wi = d["ra"].to(dtype).contiguous(), d["ri"].to(dtype).contiguous()
    c_off = -(-W // 4) * 4
    state = torch.randn(max(slots) + 2, c_off + taps * W, generator=torch.Generator().manual_seed(1)).to(DEV)
    state[slots] = 0.0
    rest = [s for s in range(state.shape[0]) if s not in slots]
    before = state[rest].clone()
    fed, got = [0] * len(xs), [[] for _ in xs]
    for step in range(max(len(c) for c in cuts)):
        live = [r for r in range(len(xs)) if step < len(cuts[r])]
        rows = [xs[r][fed[r]:fed[r] + cuts[r][step]] for r in live]
        proj = torch.cat(rows).to(DEV).contiguous()
        starts = [0]
        for r in rows:
            starts.append(starts[-1] + r.shape[0])
        qs, sl = i32(starts), i32([slots[r] for r in live])
        longest = max(r.shape[0] for r in rows)
        if decode and longest == 1 and dtype == torch.bfloat16:
            out = fn.lru_decode(proj, W + 3, 2, d["x.b"], d["conv"], d["conv.b"], d["y.b"], wr, wi, d["ra.b"], d["ri.b"],
                                d["rate"], state, 0, c_off, qs, sl, out_dtype)
        else:
            req = i32([n for n, r in enumerate(rows) for _ in range(r.shape[0])])
            u = fn.causal_conv(proj, W + 3, W, d["x.b"], d["conv"], d["conv.b"], state, c_off, qs, req, sl)
            a, x = fn.lru_gates(u, wr, wi, d["ra.b"], d["ri.b"], d["rate"])
            out = fn.lru_scan(a, x, proj, 2, d["y.b"], state, 0, qs, sl, out_dtype, segments, longest)
        for n, r in enumerate(live):
            got[r].append(out[starts[n]:starts[n + 1]].float().cpu())
            fed[r] += cuts[r][step]
    assert torch.equal(state[rest], before)
    return [torch.cat(g) for g in got]


@pytest.mark.parametrize("W,blocks,taps", [(30, 3, 3), (44, 44, 5), (36, 1, 1), (128, 2, 4), (160, 5, 8), (480, 2, 2), (66, 2, 4)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_recurrence_in_portions_and_batches(W, blocks, taps, dtype):
    """Matrices in either type give 32-bit products; portions walked, in segments, and single tokens in one launch."""
    lens = [210, 1, 40]
    p, xs, _, want = lru_case(W, blocks, taps, lens, W + taps)
    runs = [([[210], [1], [40]], False), ([[70] + [1] * 140, [1], [2, 3, 1, 9, 25]], False)]
    if dtype == torch.bfloat16:
        runs += [([[210], [1], [40]], True), ([[64, 65, 3] + [1] * 78, [1], [2, 37, 1]], True)]
    outs = []
    for cuts, seg in runs:
        got = run_lru(W, blocks, taps, p, xs, cuts, dtype, seg, [3, 0, 4])
        outs.append(got)
        for r in range(3):
            assert close(got[r], want[r], 2e-5), (cuts, seg, r)
    if dtype == torch.float32:
        assert all(torch.equal(a, b) for a, b in zip(*outs))


def test_gate_products_on_the_tensor_cores_keep_all_bits_of_their_input():
    """The recurrence's input is float: an input whose digits lie beyond bfloat16's must show in the gates."""
    W, blocks, T = 96, 2, 50
    g = torch.Generator().manual_seed(2)
    n = W // blocks
    u = torch.randn(T, W, generator=g)
    wr, wi = (bf(torch.randn(blocks, n, n, generator=g)) for _ in range(2))
    br, bi, lam = (torch.randn(W, generator=g) for _ in range(3))
    z = u.double()
    r = pd.sigmoid(pd.block_product(z, wr.double(), br.double().reshape(blocks, n)))
    i = pd.sigmoid(pd.block_product(z, wi.double(), bi.double().reshape(blocks, n)))
    log_a = -8 * r * pd.softplus(lam.double())
    want = torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a)) * i * z
    args = [t.to(DEV) for t in (br, bi, (-8 * pd.softplus(lam.double())).float())]
    got = F().lru_gates(u.to(DEV), wr.to(torch.bfloat16).to(DEV), wi.to(torch.bfloat16).to(DEV), *args)
    assert close(got[0], want[0], 3e-6) and close(got[1], want[1], 3e-6)


def test_a_channel_that_forgets_nothing_carries_its_first_drive_to_the_end():
    """lam far below zero: a is one but for a few units in the last place, and 1 - a^2 must not come out as zero."""
    W, T = 40, 500
    p, xs, _, _ = lru_case(W, 2, 2, [T], 6)
    p["lam"] = torch.full((W,), -12.0)
    p["x.b"].zero_()
    p["conv.b"].zero_()
    x = xs[0]
    x[1:, W + 3:2 * W + 3] = 0.0                              # one input at the start, silence afterwards
    z, P = x.double(), {k: v.double() for k, v in p.items()}
    u = pd.causal_conv(z[:, W + 3:2 * W + 3], P["conv"], P["conv.b"])
    r, i = (pd.sigmoid(pd.block_product(u, P[k], P[k + ".b"].reshape(2, W // 2))) for k in ("ra", "ri"))
    S = pd.real_gated_lru(u, r, i, P["lam"])
    assert float(S[T - 1].abs().max()) > 0.5 * float(S.abs().max()) > 0
    want = S * pd.gelu_tanh(z[:, 2:W + 2] + P["y.b"])
    for cuts, seg in (([T], False), ([T], True), ([300] + [1] * 200, True)):
        got = run_lru(W, 2, 2, p, [x], [cuts], torch.bfloat16, seg, [0])[0]
        assert close(got, want, 3e-5), (cuts, seg)


# --------------------------------------------------------------------------- #
# attention inside chunks with a sink and a gate per head
# --------------------------------------------------------------------------- #

def paged(k, v, page_size, seed, dtype):
    T, G, d = k.shape
    n = -(-T // page_size)
    order = torch.randperm(2 * n + 3, generator=torch.Generator().manual_seed(seed))[:n].tolist()
    kc, vc = (torch.full((2 * n + 3, G, page_size, x.shape[2]), 99.0) for x in (k, v))
    for t in range(T):
        kc[order[t // page_size], :, t % page_size] = k[t]
        vc[order[t // page_size], :, t % page_size] = v[t]
    return kc.to(dtype).to(DEV), vc.to(dtype).to(DEV), order


def plain_chunks(q, k, v, scale, chunk, sink, gate):
    T, H, d = q.shape
    G = k.shape[1]
    pos = torch.arange(T)
    vis = (pos[None, :] <= pos[:, None]) & (pos[None, :] // chunk == pos[:, None] // chunk)
    out = torch.zeros(T, H, v.shape[2], dtype=torch.float64)
    for h in range(H):
        s = (q[:, h].double() @ k[:, h // (H // G)].double().T) * scale
        out[:, h] = pd.sink_softmax(s, vis, sink[h].double()) @ v[:, h // (H // G)].double()
    return out * pd.sigmoid(gate.double())[:, :, None]


def run_chunks(q, k, v, scale, chunk, sink, gate, cuts, dtype, kernel, page_size=8):
    """The sequence's queries cut into steps; pages behind the first query's chunk are taken out of the table, as the
    cache manager gives them back.  ``kernel``: plain | mma | memory (single tokens then on the split kernels)."""
    fn = F()
    T, H, d = q.shape
    e = v.shape[2]
    kc, vc, order = paged(k, v, page_size, 5, dtype)
    gates = torch.cat([torch.zeros(T, 2), gate], dim=1).to(DEV)         # from column 2 on
    outs, lo = [], 0
    for n in cuts:
        table = list(order) + [-1] * 4
        for p in range(lo // chunk * chunk // page_size):
            table[p] = -1
        kw = dict(sink=True, chunk=chunk, sink_score=sink.to(DEV), gate=gates[lo:lo + n].contiguous(), gate_col=2)
        qq = q[lo:lo + n].to(dtype).to(DEV).contiguous()
        args = (qq, kc, vc)
        where = (i32([table]), i32([0, n]), i32([lo + n]))
        if kernel == "plain":
            got = fn.attention_mix(*args, None, *where, n, 0, scale, 0.0, **kw)
        elif n == 1 and kernel == "memory":
            splits = -(-(lo + 1) // 128)
            po, pm = torch.empty(splits * H * e, device=DEV), torch.empty(splits * H * 2, device=DEV)
            got = fn.decode_attention(*args, *where, po, pm, splits, 0, scale=scale, split=128, **kw)
        elif n == 1:
            splits = fn.attention_mix_tc_splits(min(chunk, lo + 1))
            po, pm = torch.empty(splits * H * e, device=DEV), torch.empty(splits * H * 2, device=DEV)
            got = fn.attention_mix_tc(*args, None, *where, 1, 0, scale, 0.0, splits, po, pm, **kw)
        elif kernel == "memory":
            got = fn.prefill_attention_tc(*args, *where, n, 0, scale, **kw)
        else:
            got = fn.attention_mix_tc(*args, None, *where, n, 0, scale, 0.0, **kw)
        outs.append(got.float().cpu())
        lo += n
    assert lo == T
    if kernel == "memory":
        fn.check_tc_status()
    return torch.cat(outs)


CUTS = ([300], [170] + [1] * 130, [7, 2, 130, 3, 2, 5, 17, 2, 131, 1])


@pytest.mark.parametrize("kernel,H,G,d,chunk,page", [
    ("plain", 4, 2, 12, 10, 8), ("plain", 5, 1, 34, 64, 16), ("plain", 2, 2, 96, 1, 8), ("plain", 3, 3, 130, 37, 4),
    ("mma", 4, 2, 64, 21, 8), ("mma", 6, 3, 128, 100, 16), ("mma", 2, 1, 64, 1, 8),
    ("memory", 4, 2, 64, 21, 8), ("memory", 2, 1, 128, 100, 16), ("memory", 3, 3, 128, 64, 64), ("memory", 6, 2, 64, 3, 32),
    ("memory", 2, 2, 64, 256, 16)])
def test_attention_inside_chunks_in_any_cut(kernel, H, G, d, chunk, page):
    g = torch.Generator().manual_seed(H + d + chunk)
    T, scale = 300, 2.0 * d ** -0.5
    r = lambda *s: bf(torch.randn(*s, generator=g))
    q, k, v = r(T, H, d), r(T, G, d), r(T, G, d)
    sink, gate = torch.randn(H, generator=g) * 2, torch.randn(T, H, generator=g) * 2
    want = plain_chunks(q, k, v, scale, chunk, sink, gate)
    dtype, tol = (torch.float32, 3e-6) if kernel == "plain" else (torch.bfloat16, 1.5e-2)
    for cuts in CUTS:
        assert close(run_chunks(q, k, v, scale, chunk, sink, gate, cuts, dtype, kernel, page), want, tol), cuts


@pytest.mark.parametrize("kernel,d,chunk", [("plain", 16, 9), ("plain", 16, 64), ("mma", 64, 33), ("memory", 64, 33),
                                            ("memory", 128, 96), ("memory", 64, 130)])
def test_a_key_just_inside_and_just_outside_a_chunk(kernel, d, chunk):
    """One key's score stands out by thirty.  The queries of its chunk from it on read its value and no other query does,
    whether it is a chunk's first or last key; a sink below every score changes nothing."""
    T, H = 3 * chunk + 5, 2
    dtype = torch.float32 if kernel == "plain" else torch.bfloat16
    for at in (chunk, 2 * chunk - 1, 0, chunk - 1):
        g = torch.Generator().manual_seed(at)
        q, k = torch.zeros(T, H, d), bf(torch.randn(T, 1, d, generator=g)) * 0.1
        q[:, :, 0] = 1.0
        k[:, :, 0] = 0.0
        k[at, 0, 0] = 30.0
        v = bf(torch.randn(T, 1, d, generator=g)) * 0.1
        v[at, 0] = 5.0
        sink, gate = torch.full((H,), -20.0), torch.full((T, H), 30.0)
        for cuts in ([T], [at + 1] + [1] * (T - at - 1) if at + 1 < T else [T], [2] * (T // 2) + ([1] if T % 2 else [])):
            got = run_chunks(q, k, v, 1.0, chunk, sink, gate, cuts, dtype, kernel)
            sees = torch.tensor([at <= t and t // chunk == at // chunk for t in range(T)])
            assert bool(((got[:, :, 0] > 4.9) == sees[:, None]).all()), (at, cuts[:3])
            assert bool((got[~sees].abs() < 1.0).all())


@pytest.mark.parametrize("kernel,d", [("plain", 16), ("mma", 64), ("memory", 64)])
def test_a_sink_takes_its_share_once_and_is_not_scaled(kernel, d):
    """Equal scores of zero: with m keys in sight a head's output is m / (m + e^sink) of the value."""
    T, chunk = 140, 70
    sink, gate = torch.tensor([-30.0, 0.0, 3.0, 30.0]), torch.full((T, 4), 40.0)
    q, k, v = torch.zeros(T, 4, d), torch.zeros(T, 1, d), torch.ones(T, 1, d)
    m = torch.tensor([t % chunk + 1.0 for t in range(T)]).double()
    want = m[:, None] / (m[:, None] + torch.exp(sink.double())[None, :])
    for cuts in ([T], [75] + [1] * 65):
        got = run_chunks(q, k, v, 0.01, chunk, sink, gate, cuts, torch.float32 if kernel == "plain" else torch.bfloat16, kernel)
        assert float((got.double() - want[:, :, None]).abs().max()) <= (3e-6 if kernel == "plain" else 6e-3), cuts


def test_unequal_requests_in_one_step_of_chunk_attention():
    """Three requests at unlike positions in their chunks, one bringing a single token, against each alone."""
    fn = F()
    g = torch.Generator().manual_seed(3)
    H, G, d, chunk, page = 4, 2, 64, 50, 16
    totals, news = [130, 61, 49], [70, 1, 49]
    sink = torch.randn(H, generator=g)
    per = [(bf(torch.randn(n, H, d, generator=g)), bf(torch.randn(n, G, d, generator=g)), bf(torch.randn(n, G, d, generator=g)),
            torch.randn(n, H, generator=g)) for n in totals]
    for kernel, dtype, tol in (("plain", torch.float32, 3e-6), ("memory", torch.bfloat16, 1.5e-2), ("mma", torch.bfloat16, 1.5e-2)):
        tables, kcs, vcs, base = [], [], [], 0
        for q, k, v, _ in per:
            kc, vc, order = paged(k, v, page, 7, dtype)
            tables.append([base + o for o in order] + [-1] * (10 - len(order)))
            kcs.append(kc)
            vcs.append(vc)
            base += kc.shape[0]
        kc, vc = torch.cat(kcs), torch.cat(vcs)
        q = torch.cat([p[0][-n:] for p, n in zip(per, news)]).to(dtype).to(DEV)
        gate = torch.cat([p[3][-n:] for p, n in zip(per, news)]).to(DEV)
        where = (i32(tables), i32([0, 70, 71, 120]), i32(totals))
        kw = dict(sink=True, chunk=chunk, sink_score=sink.to(DEV), gate=gate)
        if kernel == "plain":
            got = fn.attention_mix(q, kc, vc, None, *where, 70, 0, 0.2, 0.0, **kw)
        elif kernel == "memory":
            got = fn.prefill_attention_tc(q, kc, vc, *where, 70, 0, 0.2, **kw)
        else:
            got = fn.attention_mix_tc(q, kc, vc, None, *where, 70, 0, 0.2, 0.0, **kw)
        want = torch.cat([plain_chunks(*p[:3], 0.2, chunk, sink, p[3])[-n:] for p, n in zip(per, news)])
        assert close(got.float(), want, tol), kernel


@pytest.mark.parametrize("H,G,d", [(64, 64, 128), (160, 4, 32), (96, 24, 200)])
def test_more_heads_than_one_block_holds(H, G, d):
    """Heads that exchange nothing are shared out over blocks (float32)."""
    assert not F().attention_mix_supported(H, G, d, d, torch.float32)
    assert F().attention_mix_supported(H, G, d, d, torch.float32, independent=True)
    g = torch.Generator().manual_seed(H)
    T = 40
    q, k, v = (torch.randn(T, n, d, generator=g) for n in (H, G, G))
    sink, gate = torch.randn(H, generator=g), torch.randn(T, H, generator=g)
    want = plain_chunks(q, k, v, d ** -0.5, 13, sink, gate)
    for cuts in ([T], [30] + [1] * 10):
        assert close(run_chunks(q, k, v, d ** -0.5, 13, sink, gate, cuts, torch.float32, "plain"), want, 3e-6), cuts


# --------------------------------------------------------------------------- #
# rotation, head norms behind it, keys as values
# --------------------------------------------------------------------------- #

@pytest.mark.parametrize("H,G,d,rot", [(4, 2, 12, 8), (3, 1, 34, 6), (2, 2, 128, 32), (8, 4, 64, 64), (2, 1, 256, 20), (5, 5, 16, 0),
                                       (1, 1, 10, 10)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_biased_rotated_normalised_heads_with_keys_as_values(H, G, d, rot, dtype):
    from mini_infer_b200.config.registry import part_class
    g = torch.Generator().manual_seed(H + d + rot)
    T, page, eps = 37, 8, 1e-5
    width = (H + G) * d
    x, bias = torch.randn(T, width + H, generator=g), torch.randn(width, generator=g) * 0.5
    rows = {"dims": rot, "base": 2000.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    pos = torch.arange(5, 5 + T)
    z = (x[:, :width] + bias).double()
    q, k = z[:, :H * d].reshape(T, H, d), z[:, H * d:].reshape(T, G, d)
    want_q, want_k = (pd.unit_rms(pd.rotate_neighbours(a, pos, rows), eps) for a in (q, k))
    table, mag = None, 1.0
    if rot:
        part = part_class("position", "rope_yarn")({"head_dim": d, "rot_dim": rot, "theta": 2000.0, "pairing": "neighbours",
                                                     "factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0})
        table, mag = part.table(DEV), part.magnitude
    kc, vc = torch.zeros(8, G, page, d, dtype=dtype, device=DEV), torch.zeros(8, G, page, d, dtype=dtype, device=DEV)
    slots = list(range(11, 11 + T))
    slots[3] = -1                                              # written nowhere
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    for pad in (0, 1):                                          # rows on 16-byte boundaries or not
        xx = torch.cat([x, torch.zeros(T, (-x.shape[1]) % 4 + pad)], dim=1).to(DEV).contiguous()
        got = F().rope_store(xx, i32(pos.tolist()), table, rot, i32(slots), kc, vc, H, G, d, d, page, dtype, eps=eps,
                             neighbours=True, bias=bias.to(DEV), values_are_keys=True, norm="after", magnitude=mag)
        assert close(got.float(), want_q, tol)
        for cache, want in ((kc, want_k), (vc, k)):
            flat = cache.float().cpu().permute(0, 2, 1, 3).reshape(-1, G, d)
            assert bool((flat[14] == 0).all())                  # the slot it would have had
            keep = [t for t in range(T) if slots[t] >= 0]
            assert close(flat[[slots[t] for t in keep]], want[keep], tol)


@pytest.mark.parametrize("neighbours", [True, False])
@pytest.mark.parametrize("d,rot", [(12, 8), (16, 16), (34, 6)])
def test_head_norm_with_gains_behind_the_rotation_and_own_values(neighbours, d, rot):
    g = torch.Generator().manual_seed(d)
    T, H, G, dv, page = 9, 3, 1, 10, 4
    x = torch.randn(T, (H + G) * d + G * dv, generator=g)
    bias = torch.randn((H + G) * d + G * dv, generator=g)
    gq, gk = 1 + 0.3 * torch.randn(d, generator=g), 1 + 0.3 * torch.randn(d, generator=g)
    z = (x + bias).double()
    half = rot // 2
    freq = torch.tensor([100.0 ** (-2 * i / rot) for i in range(half)], dtype=torch.float64)

    def turn(a):
        ang = torch.arange(T).double()[:, None] * freq
        c, s = 1.3 * torch.cos(ang)[:, None], 1.3 * torch.sin(ang)[:, None]
        u, v = (a[..., 0:rot:2], a[..., 1:rot:2]) if neighbours else (a[..., :half], a[..., half:rot])
        out = a.clone()
        if neighbours:
            out[..., 0:rot:2], out[..., 1:rot:2] = u * c - v * s, v * c + u * s
        else:
            out[..., :half], out[..., half:rot] = u * c - v * s, v * c + u * s
        return out

    want_q = pd.unit_rms(turn(z[:, :H * d].reshape(T, H, d)), 1e-6) * gq.double()
    want_k = pd.unit_rms(turn(z[:, H * d:(H + G) * d].reshape(T, G, d)), 1e-6) * gk.double()
    kc, vc = torch.zeros(4, G, page, d, device=DEV), torch.zeros(4, G, page, dv, device=DEV)
    got = F().rope_store(x.to(DEV), i32(list(range(T))), freq.float().to(DEV), rot, i32(list(range(T))), kc, vc, H, G, d, dv, page,
                         torch.float32, gq.to(DEV), gk.to(DEV), 1e-6, neighbours=neighbours, bias=bias.to(DEV), norm="after",
                         magnitude=1.3)
    assert close(got, want_q, 3e-6)
    assert close(kc.cpu().permute(0, 2, 1, 3).reshape(-1, G, d)[:T], want_k, 3e-6)
    assert close(vc.cpu().permute(0, 2, 1, 3).reshape(-1, G, dv)[:T], z[:, (H + G) * d:].reshape(T, G, dv), 1e-6)


# --------------------------------------------------------------------------- #
# pairs of normalised outputs, squared rectifier
# --------------------------------------------------------------------------- #

@pytest.mark.parametrize("T,W", [(1, 40), (7, 192), (5, 33), (3, 1026), (2, 4100), (2, 8192), (2, 9000), (300, 64)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_two_normalised_outputs_join_the_residual(T, W, dtype):
    g = torch.Generator().manual_seed(T + W)
    h, y1, y2 = torch.randn(T, W, generator=g), torch.randn(T, W, generator=g) * 3, torch.randn(T, W, generator=g) * 0.1
    w1, w2, w = (1 + 0.3 * torch.randn(W, generator=g) for _ in range(3))
    new = h.double() + 0.5 * pd.unit_rms(y1.double(), 1e-5) * w1.double() + 0.7 * pd.unit_rms(y2.double(), 1e-6) * w2.double()
    want = pd.unit_rms(new, 1e-5) * w.double()
    pair = ((y1.to(DEV), w1.to(DEV), 0.5, 1e-5), (y2.to(DEV), w2.to(DEV), 0.7, 1e-6))
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    hidden = h.to(DEV)
    assert F().normed_pair_add(hidden, pair) is None and close(hidden, new, 3e-6)
    for weight in (w.to(DEV), w.to(torch.bfloat16).to(DEV)):
        hidden = h.to(DEV)
        x = F().normed_pair_add(hidden, pair, weight, 1e-5, dtype)
        assert close(hidden, new, 3e-6) and close(x.float(), pd.unit_rms(new, 1e-5) * weight.cpu().double(), tol)
    hidden, rows = h.to(DEV), [T - 1, 0]
    x = F().normed_pair_add(hidden, pair, w.to(DEV), 1e-5, dtype, i32(rows))
    assert torch.equal(hidden.cpu(), h) and close(x.float(), want[rows], tol)


@pytest.mark.parametrize("n,gate_dtype", [(40, torch.float32), (96, torch.bfloat16), (33, torch.bfloat16), (2048, torch.float32)])
def test_norm_of_all_heads_together_with_its_gate(n, gate_dtype):
    g = torch.Generator().manual_seed(n)
    T = 7
    o, gate, w = torch.randn(T, n, generator=g) * 3, bf(torch.randn(T, n + 3, generator=g)), 1 + 0.2 * torch.randn(n, generator=g)
    want = pd.unit_rms(o.double(), 1e-5) * w.double() * pd.sigmoid(gate[:, 1:n + 1].double())
    got = F().memory_finish(o.to(DEV), gate.to(gate_dtype).to(DEV), 1, w.to(DEV), 1e-5, torch.float32)
    assert close(got, want, 3e-6)


@pytest.mark.parametrize("T,n", [(1, 33), (5, 64), (40, 100)])
def test_squared_rectifier(T, n):
    g = torch.Generator().manual_seed(n)
    x = torch.randn(T, n, generator=g)
    assert close(F().squared_relu_(x.clone().to(DEV)), torch.relu(x.double()) ** 2, 1e-6)
    xb = bf(x)
    assert close(F().squared_relu_(xb.to(torch.bfloat16).to(DEV)).float(), torch.relu(xb.double()) ** 2, 8e-3)
    if T <= 32:
        a, w = bf(torch.randn(T, 96, generator=g)), bf(torch.randn(n, 96, generator=g))
        got = F().dense_skinny(a.to(torch.bfloat16).to(DEV), w.to(torch.bfloat16).to(DEV), squared_relu=True)
        assert close(got.float(), torch.relu(a.double() @ w.double().T) ** 2, 8e-3)
