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
            f = pd.log_sigmoid(c * torch.tanh((z[:, extra["col_i"] + H:] + extra["bf"].double()) / c))
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
        starts = [0]
        for r in rows:
            starts.append(starts[-1] + r.shape[0])
        args = (proj, extra["cols"], st, state, i32(starts), i32([slots[r] for r in live]))
        longest = max(r.shape[0] for r in rows)
        if decode and longest == 1:
            y = fn.memory_decode(*args, gate_col=extra["col_g"], weight=extra["w"].to(DEV), eps=1e-5, out_dtype=dtype, **kw)
        else:
            y = fn.memory_scan(*args, chunks=chunks, max_q_len=longest, **kw)
            if log_gates:
                y = fn.memory_finish(*y, proj, extra["col_g"], extra["w"].to(DEV), 1e-5, dtype)
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
def test_memory_in_chunks_and_decoded(H, d, dv, log_gates):
    """Long portions over chunks of 64 tokens, portions that end inside a chunk, single tokens on the decode kernel.  The
    projections are bfloat16 numbers already, so the forms differ from the plain sums by what float and a pair of bfloat16
    lose only (silu, whose result the chunks round to bfloat16, aside)."""
    lens = [300, 1, 70, 65]
    xs, want, extra = memory_case(H, d, dv, lens, 7 * H + d + dv, log_gates)
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
        x[:, extra["col_i"] + H:] = 8.0                             # forget gates near one
        i = extra["cap"] * torch.tanh((x[:, extra["col_i"]:extra["col_i"] + H].double() + extra["bi"].double()) / extra["cap"])
        f = pd.log_sigmoid(extra["cap"] * torch.tanh((x[:, extra["col_i"] + H:].double() + extra["bf"].double()) / extra["cap"]))
        z = x.double()
        o = pd.matrix_memory(z[:, c[0]:c[0] + H * d].reshape(T, H, d) * d ** -0.5, z[:, c[1]:c[1] + H * d].reshape(T, H, d),
                             z[:, c[2]:c[2] + H * dv].reshape(T, H, dv), i, f)
        want = pd.unit_rms(o, 1e-5).reshape(T, H * dv) * extra["w"].double() * pd.sigmoid(z[:, extra["col_g"]:extra["col_g"] + H * dv])
    else:
        extra["decay"] = torch.tensor([1.0, 0.999])
        z = pd.silu(x.double())
        want = pd.fixed_decay_memory(*(z[:, a:a + H * n].reshape(T, H, n) for a, n in zip(c, (d, d, dv))),
                                     extra["decay"].double()).reshape(T, H * dv)
        v5 = z[5, c[2]:c[2] + H * dv]
        assert float((want[T - 1] - v5 * 0).abs().max()) > 10                # the far value is what is read
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
    x[:, ci + H:] = bf(torch.randn(T, H, generator=g) * 20)
    x[100:180, ci + H:] = -60.0                                     # forget everything at every token
    x[180:, ci:ci + H] = -60.0                                      # and write next to nothing
    z = x.double()
    i = 15 * torch.tanh((z[:, ci:ci + H] + extra["bi"].double()) / 15)
    f = pd.log_sigmoid(15 * torch.tanh((z[:, ci + H:] + extra["bf"].double()) / 15))
    o = pd.matrix_memory(z[:, c[0]:c[0] + H * d].reshape(T, H, d) * d ** -0.5, z[:, c[1]:c[1] + H * d].reshape(T, H, d),
                         z[:, c[2]:c[2] + H * dv].reshape(T, H, dv), i, f)
    want = pd.unit_rms(o, 1e-5).reshape(T, H * dv) * extra["w"].double() * pd.sigmoid(z[:, extra["col_g"]:extra["col_g"] + H * dv])
    for cuts, chunks in (([T], False), ([T], True), ([130] + [1] * 130, True)):
        got = run_memory(H, d, dv, [x], extra, [cuts], True, chunks, torch.float32)[0]
        assert bool(torch.isfinite(got).all())
        err = (got.double() - want).abs().max(dim=1).values / want.abs().max()
        assert float(err.max()) <= 2e-3 and float(err.median()) <= 2e-5, (cuts, chunks, float(err.max()))
