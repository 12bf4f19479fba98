"""The kernels that Gedilorn added or widened, each against the plain function of the same mechanism (float64 on the
CPU), on sizes the tiny models do not reach, cut into portions and decoded, over hand-made paged caches, with inputs
made so that one key stands out at a page's or a key tile's edge and just inside and just outside a window."""

import pytest
import torch

import plain_gedilorn as pg

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BF, F32 = torch.bfloat16, torch.float32
TOL = {F32: 2e-5, BF: 1.5e-2}


def F():
    from mini_infer_b200.ops import functional
    return functional


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def close(got, want, tol, what=""):
    err = float((got.double().cpu() - want).abs().max())
    assert err <= tol * float(want.abs().max()), f"{what}: {err:.2e} of {float(want.abs().max()):.2e}"


# --------------------------------------------------------------------------- #
# embedding
# --------------------------------------------------------------------------- #

@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("W,S,buckets,mp,mc", [(48, 2, 37, 31, 7), (50, 1, 1, 5, 3), (1028, 4, 4001, 2 ** 31 + 11, 2 ** 33 + 5),
                                               (256, 7, 12, 0, 1)])
def test_embedding_with_a_second_table_in_any_cut(dtype, W, S, buckets, mp, mc):
    """Three requests whose portions are cut anywhere, so that the token before a portion's first one lies in a page of
    its own request (page edges included)."""
    g = torch.Generator().manual_seed(W)
    V, ps = 97, 4
    w = {"embed": torch.randn(V, W, generator=g).to(dtype), "bigram": torch.randn(buckets + 1, W, generator=g).to(dtype),
         "embed.norm": 1.0 + 0.2 * torch.randn(W, generator=g)}
    cfg = {"embedding": {"scale": 2.5, "bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}, "norm": {"eps": 1e-6}}
    toks = [torch.randint(0, V, (n,), generator=g).tolist() for n in (13, 6, 9)]
    want = [pg.embedding_output(cfg, {k: v.double() for k, v in w.items()}, t) for t in toks]
    dev = {k: v.to(DEV) for k, v in w.items()}
    pages = torch.randperm(16, generator=g).tolist()
    tables = [[pages.pop() for _ in range(4)] for _ in toks]
    ids = torch.full((16, ps), -7, dtype=torch.int32, device=DEV)
    fed = [0, 0, 0]
    for step in ([(0, 4), (1, 1)], [(2, 2), (0, 1), (1, 3)], [(0, 3), (2, 7), (1, 2)], [(0, 1)], [(0, 4)]):
        flat, pos, req, slot, rows = [], [], [], [], []
        for b, (r, n) in enumerate(step):
            for p in range(fed[r], fed[r] + n):
                flat.append(toks[r][p]); pos.append(p); req.append(b); rows.append((r, p))
                slot.append(tables[r][p // ps] * ps + p % ps)
            fed[r] += n
        bigram = (dev["bigram"], buckets, mp, mc, i32(pos), i32(req), ids, i32([tables[r] for r, _ in step]), i32(slot))
        got = F().streams_embed(i32(flat), dev["embed"], 2.5, S, (dev["embed.norm"], 1e-6), bigram)
        assert got.shape == (len(flat), S, W)
        for s in range(S):
            close(got[:, s], torch.stack([want[r][p] for r, p in rows]), 1e-5, f"stream {s}")
    assert fed == [13, 6, 9]


def test_embedding_rows_of_no_request_write_no_token_id_and_a_norm_is_optional():
    table = torch.randn(5, 12, device=DEV)
    second = torch.randn(4, 12, device=DEV)
    ids = torch.full((2, 4), -7, dtype=torch.int32, device=DEV)
    got = F().streams_embed(i32([3, 0]), table, 0.5, 1, None, (second, 3, 2, 1, i32([0, 0]), i32([0, 1]), ids,
                                                               i32([[1], [0]]), i32([4, -1])))
    close(got[:, 0], (table[[3, 0]] * 0.5 + second[[3, 3]]).double().cpu(), 1e-6)
    assert ids.flatten().tolist() == [-7] * 4 + [3] + [-7] * 3
    close(F().streams_embed(i32([2]), table, 3.0, 2)[:, 1], table[2:3].double().cpu() * 3.0, 1e-6)


# --------------------------------------------------------------------------- #
# residual streams
# --------------------------------------------------------------------------- #

@pytest.mark.parametrize("out", [F32, BF])
@pytest.mark.parametrize("S,W", [(1, 48), (2, 50), (3, 256), (4, 1028), (3, 2052), (2, 4096), (3, 5000), (6, 54), (9, 1024)])
def test_streams_update_and_read(out, S, W):
    T, eps = 5, 1e-5
    g = torch.Generator().manual_seed(S * W)
    xs, y = torch.randn(T, S, W, generator=g), torch.randn(T, W, generator=g)
    mix, wo, wi = (torch.randn(S, S, generator=g), torch.randn(S, generator=g), torch.randn(S, generator=g))
    gain = (1.0 + 0.2 * torch.randn(W, generator=g)).to(out)
    d = lambda t: t.to(DEV)
    new = pg.streams_update(xs.double(), mix.double(), wo.double(), y.double())
    norm = lambda x: pg.rms_norm(pg.streams_read(x, wi.double()), gain.double(), eps)
    tol = 1e-5 if out == F32 else 5e-3
    # nothing pending: the streams are read as they are
    x = d(xs)
    close(F().streams_read(x, None, d(wi), d(gain), eps, out), norm(xs.double()), tol)
    assert torch.equal(x, d(xs))
    # chosen rows, in any order and twice: the streams are left alone
    rows = [3, 0, 3]
    close(F().streams_read(x, (d(y), d(mix), d(wo)), d(wi), d(gain), eps, out, i32(rows)), norm(new)[rows], tol)
    assert torch.equal(x, d(xs))
    close(F().streams_sum(x, (d(y), d(mix), d(wo))), new.sum(1), 1e-5)
    close(F().streams_sum(x), xs.double().sum(1), 1e-5)
    assert torch.equal(x, d(xs))
    # the update: all streams at once from the old ones
    whole = F().streams_read(x, (d(y), d(mix), d(wo)), d(wi), d(gain), eps, out)
    close(whole, norm(new), tol)
    close(x, new, 1e-5)
    # a row alone or among others: no bit moves
    one = d(xs)[2:3].contiguous()
    assert torch.equal(F().streams_read(one, (d(y)[2:3].contiguous(), d(mix), d(wo)), d(wi), d(gain), eps, out)[0], whole[2])
    assert torch.equal(one[0], x[2])


# --------------------------------------------------------------------------- #
# feed-forward with a rectified gate
# --------------------------------------------------------------------------- #

@pytest.mark.parametrize("T,I", [(1, 8), (7, 33), (130, 96), (3, 4096)])
def test_relu_glu(T, I):
    g = torch.Generator().manual_seed(I)
    gu = torch.randn(T, 2 * I, generator=g)
    for dtype in (F32, BF):
        x = gu.to(dtype)
        want = torch.relu(x.double()[:, :I]) * x.double()[:, I:]
        close(F().relu_glu(x.to(DEV)), want, 1e-6 if dtype == F32 else 5e-3)


@pytest.mark.parametrize("T,K,I", [(1, 32, 16), (8, 96, 40), (15, 1056, 72), (32, 64, 24)])
def test_gate_and_up_product_of_small_steps_with_a_rectified_gate(T, K, I):
    g = torch.Generator().manual_seed(T + I)
    x, w = torch.randn(T, K, generator=g).to(BF), (torch.randn(2 * I, K, generator=g) * 0.2).to(BF)
    gu = x.double() @ w.double().T
    got = F().dense_skinny(x.to(DEV), w.to(DEV), swiglu_pair=True, activation="relu")
    close(got, torch.relu(gu[:, :I]) * gu[:, I:], 1e-2)


# --------------------------------------------------------------------------- #
# attention of (query, head) rows over one shared key/value head
# --------------------------------------------------------------------------- #

def plain_shared(q, rows, c, window, scale):
    """``q [T, H, dk]``, ``rows [T, dk]`` -> ``[T, H, c]``."""
    T, H, _ = q.shape
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    mask = (j <= i) & ((i - j < window) if window else torch.ones(T, T, dtype=torch.bool))
    s = torch.einsum("thd,jd->htj", q, rows) * scale
    p = torch.softmax(s.masked_fill(~mask, float("-inf")), dim=-1)
    return torch.einsum("htj,jc->thc", p, rows[:, :c])


def paged_rows(rows, page_size, num_pages, seed, dtype, drop=()):
    """``rows [T, dk]`` over pages in a shuffled order; memory that belongs to no row holds large numbers."""
    T, dk = rows.shape
    n = -(-T // page_size)
    order = torch.randperm(num_pages, generator=torch.Generator().manual_seed(seed))[:n].tolist()
    cache = torch.full((num_pages, 1, page_size, dk), 99.0)
    for t in range(T):
        if t // page_size not in drop:
            cache[order[t // page_size], 0, t % page_size] = rows[t]
    return cache.to(dtype).to(DEV), [-1 if i in drop else p for i, p in enumerate(order)]


def shared(form, q, cache, table, q_start, kv_len, max_q, window, scale, c, splits=1):
    args = (q, cache, i32(table), i32(q_start), i32(kv_len), max_q, window, scale, c)
    return F().attention_shared_plain(*args) if form == "plain" else F().attention_shared_tc(*args, splits=splits)


SHARED_SIZES = [(3, 40, 24, 0), (16, 128, 16, 0), (36, 64, 8, 9), (1, 8, 8, 1), (40, 256, 32, 64), (5, 512, 64, 0), (128, 136, 16, 33),
                (20, 96, 40, 257)]


@pytest.mark.parametrize("H,c,r,window", SHARED_SIZES)
@pytest.mark.parametrize("form", ["tc", "plain", "plain32"])
def test_shared_head_attention_in_any_cut(form, H, c, r, window):
    T, ps, scale = 150, 8, 0.2
    dtype = F32 if form == "plain32" else BF
    kind = "tc" if form == "tc" else "plain"
    g = torch.Generator().manual_seed(H + c)
    rows = (torch.randn(T, c + r, generator=g) * 0.7).to(dtype).float()
    q = (torch.randn(T, H, c + r, generator=g) * 0.5).to(dtype).float()
    want = plain_shared(q.double(), rows.double(), c, window, scale)
    whole = None
    for cuts in ([T], [1, 2, 60, 1, 64, 2, 1, 19], [147, 1, 1, 1]):
        assert sum(cuts) == T
        lo, outs = 0, []
        for n in cuts:
            # pages that no remaining query sees are given back
            drop = set(range(max(0, lo - window + 1) // ps)) if window else ()
            cache, table = paged_rows(rows[:lo + n], ps, 30, 3, dtype, drop)
            splits = 1 if n > 2 else (lo % 5) + 1
            outs.append(shared(kind, q[lo:lo + n].to(dtype).to(DEV).contiguous(), cache, [table], [0, n], [lo + n], n,
                               window, scale, c, splits).float().cpu())
            lo += n
        got = torch.cat(outs)
        close(got, want, TOL[dtype], f"{cuts}")
        if form == "plain32":
            whole = got if whole is None else whole
            assert torch.equal(got, whole)              # no bit moves


@pytest.mark.parametrize("form", ["tc", "plain"])
def test_shared_head_attention_of_odd_sizes_and_unequal_requests(form):
    """Requests of one token and of many in one call, over one cache, with sizes that are no multiples of eight for
    the plain form; a request alone gives the same as in the batch."""
    H, c, r, ps = (6, 40, 8, 16) if form == "tc" else (3, 13, 6, 4)
    dtype, scale = (BF if form == "tc" else F32), 0.3
    g = torch.Generator().manual_seed(1)
    lens, new = [70, 1, 33, 130], [1, 1, 20, 67]
    pool = torch.full((80, 1, ps, c + r), 55.0)
    order = torch.randperm(80, generator=g).tolist()
    tables, qs, wants = [], [], []
    for L, n in zip(lens, new):
        rows = torch.randn(L, c + r, generator=g).to(dtype).float()
        q = torch.randn(L, H, c + r, generator=g).to(dtype).float()
        t = [order.pop() for _ in range(-(-L // ps))]
        for i in range(L):
            pool[t[i // ps], 0, i % ps] = rows[i]
        tables.append(t + [-1] * (40 - len(t)))
        qs.append(q[L - n:])
        wants.append(plain_shared(q.double(), rows.double(), c, 0, scale)[L - n:])
    cache = pool.to(dtype).to(DEV)
    starts = [0, 1, 2, 22, 89]
    for splits in ((1, 3) if form == "tc" else (1,)):
        got = shared(form, torch.cat(qs).to(dtype).to(DEV), cache, tables, starts, lens, 67, 0, scale, c, splits)
        close(got, torch.cat(wants), TOL[dtype])
    for b in range(4):
        one = shared(form, qs[b].to(dtype).to(DEV), cache, tables[b:b + 1], [0, new[b]], lens[b:b + 1], new[b], 0, scale, c)
        close(one, wants[b], TOL[dtype])
        if form == "plain":
            assert torch.equal(one, got[starts[b]:starts[b + 1]])


@pytest.mark.parametrize("window", [0, 1, 7, 64, 65, 257])
@pytest.mark.parametrize("form", ["tc", "plain"])
def test_a_key_that_stands_out_far_away_and_at_every_edge(form, window):
    """One key matches the last query far better than all others: its value comes back if the query sees it, and
    leaves no trace if it lies just outside the window.  Keys at page edges, tile edges, the first key, the query's
    own; decoded (split or not) and as the end of a portion."""
    T, H, c, r, ps = 700, 4, 64, 16, 16
    g = torch.Generator().manual_seed(window)
    base = torch.randn(T, c + r, generator=g) * 0.05
    base[:, 0] = 0.0
    keys = [0, 1, 15, 16, 63, 64, 255, 256, 639, 640, 698, 699]
    if window:
        keys += [T - window, T - window - 1]
    for key in sorted({k for k in keys if 0 <= k < T}):
        rows = base.clone()
        rows[key, 0] = 6.0
        rows[key, 1] = 3.0
        rows = rows.to(BF).float()
        q = torch.zeros(T, H, c + r)
        q[-1, :, 0] = 6.0
        want = plain_shared(q.double(), rows.double(), c, window, 1.0)[-1:]
        seen = key < T and (not window or key >= T - window)
        assert (float(want[0, 0, 1]) > 2.5) == seen
        cache, table = paged_rows(rows, ps, 60, 5, BF)
        for n, splits in ((1, 1), (1, 9), (40, 1)):
            got = shared(form, q[T - n:].to(BF).to(DEV).contiguous(), cache, [table], [0, n], [T], n, window, 1.0, c, splits)
            close(got[-1:], want, 2e-2, f"key {key}, {n} queries, {splits} splits")


@pytest.mark.parametrize("H,d,r,e,c,gated", [(3, 8, 16, 12, 24, True), (16, 64, 32, 64, 128, False), (2, 130, 64, 100, 512, True),
                                             (5, 24, 8, 41, 40, True), (1, 8, 8, 8, 8, False)])
@pytest.mark.parametrize("T", [1, 3, 8, 16])
def test_folding_and_values_of_small_steps(H, d, r, e, c, gated, T):
    """``latent_fold`` (queries, rotation, cached rows), the split attention's partial results and ``latent_values``."""
    g = torch.Generator().manual_seed(H * 7 + c)
    f, mag = pg.yarn_frequencies(r, 500.0, {"factor": 8.0, "original": 64, "fast": 8.0, "slow": 0.5})
    inv = torch.tensor(f).float().to(DEV)
    ld = 3 + H * e + c + r + H * (d + r)
    y = torch.randn(T, ld, generator=g)
    gcol, kcol, qcol = 3, 3 + H * e, 3 + H * e + c + r
    w_uk, w_uv = (torch.randn(H, d, c, generator=g) * d ** -0.5).to(BF), (torch.randn(H, e, c, generator=g) * c ** -0.5).to(BF)
    gain = 1.0 + 0.1 * torch.randn(c, generator=g)
    ps = 8
    cache = torch.zeros(6, 1, ps, c + r, dtype=BF, device=DEV)
    order = torch.randperm(6, generator=g).tolist()
    slots = [order[t // ps] * ps + t % ps for t in range(T)]
    if T > 1:
        slots[1] = -1                                   # a row of no request
    yd = y.to(DEV)
    q_full = F().latent_fold(yd, qcol, H, d, w_uk.to(DEV), i32(list(range(T))), inv, r, mag,
                             (yd, kcol, gain.to(DEV), 1e-6, i32(slots), cache))
    q = y.double()[:, qcol:].view(T, H, d + r)
    want_q = torch.cat([torch.einsum("thd,hdc->thc", q[..., :d], w_uk.double()), pg.rotate_neighbours(q[..., d:], f, mag)], -1)
    close(q_full, want_q, 1e-2)
    x = y.double()[:, kcol:kcol + c + r]
    rows = torch.cat([pg.rms_norm(x[:, :c], gain.double(), 1e-6), pg.rotate_neighbours(x[:, None, c:], f, mag)[:, 0]], -1)
    for t in range(T):
        if slots[t] >= 0:
            close(cache[slots[t] // ps, 0, slots[t] % ps], rows[t], 1e-2)
    assert int((cache != 0).any(dim=-1).sum()) == sum(s >= 0 for s in slots)
    # the same queries over a context of 200 rows (a token of its own for every request), five splits
    L, ctx_rows = 200, (torch.randn(200, c + r, generator=g) * 0.5).to(BF).float()
    kc, table = paged_rows(ctx_rows, ps, 40, 2, BF)
    lens = [L - 3 * t if t < 12 else 5 for t in range(T)]
    po, pm = F().attention_shared_tc(q_full, kc, i32([table] * T), i32(list(range(T + 1))), i32(lens), 1, 0, 0.1, c,
                                     splits=5, partial=True)
    assert po.shape == (5, T * H, c)
    out = torch.full((T, H * e), 9.0, dtype=BF, device=DEV)
    F().latent_values(po, pm, w_uv.to(DEV), yd if gated else None, gcol, out)
    want = []
    for t in range(T):
        s = torch.softmax(q_full[t].double().cpu() @ ctx_rows[:lens[t]].double().T * 0.1, dim=-1)
        v = torch.einsum("hc,hec->he", s @ ctx_rows[:lens[t], :c].double(), w_uv.double()).reshape(-1)
        want.append(v * torch.sigmoid(y.double()[t, gcol:gcol + H * e]) if gated else v)
    close(out, torch.stack(want), 1.5e-2)


# --------------------------------------------------------------------------- #
# row-wise work of larger steps, keys and values formed from latents
# --------------------------------------------------------------------------- #

@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,d,r,c", [(3, 8, 4, 20), (5, 24, 8, 48), (16, 136, 40, 96), (1, 10, 2, 7)])
def test_cached_rows_and_padded_queries_in_one_launch(dtype, H, d, r, c):
    T, ps = 37, 4
    g = torch.Generator().manual_seed(d)
    f, mag = pg.yarn_frequencies(r, 100.0, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5})
    y = torch.randn(T, 5 + c + r + H * (d + r), generator=g)
    gain = 1.0 + 0.2 * torch.randn(c, generator=g)
    slots = torch.randperm(12 * ps, generator=g)[:T]
    slots[4] = -1
    cache = torch.zeros(12, 1, ps, c + r, dtype=dtype, device=DEV)
    cols, at = F().unfolded_query_layout(d, r)
    pad = torch.full((T, H, cols), 7.0, dtype=dtype, device=DEV)
    dp, rp = -(-d // 16) * 16, -(-r // 16) * 16
    yd = y.to(DEV)
    F().latent_rows(i32([3 * t for t in range(T)]), torch.tensor(f).float().to(DEV), c, r,
                    store=(yd, 5, gain.to(DEV), 1e-6, i32(slots.tolist()), cache),
                    query=(yd, 5 + c + r, H, d, pad, dp, pad, at, rp), magnitude=mag)

    def turned(x):                      # positions 0, 3, 6, ...
        full = torch.zeros(3 * T, x.shape[1], r, dtype=torch.float64)
        full[::3][:T] = x
        return pg.rotate_neighbours(full, f, mag)[::3][:T]
    tol = 1e-5 if dtype == F32 else 1e-2
    q = y.double()[:, 5 + c + r:].view(T, H, d + r)
    close(pad[..., :d], q[..., :d], tol)
    close(pad[..., at:at + r], turned(q[..., d:]), tol)
    assert float(pad[..., d:dp].float().abs().sum()) == 0.0 and float(pad[..., at + r:at + rp].float().abs().sum()) == 0.0
    x = y.double()[:, 5:5 + c + r]
    rows = torch.cat([pg.rms_norm(x[:, :c], gain.double(), 1e-6), turned(x[:, None, c:])[:, 0]], -1)
    for t in range(T):
        s = int(slots[t])
        if s >= 0:
            close(cache[s // ps, 0, s % ps], rows[t], tol)
    assert int((cache != 0).any(dim=-1).sum()) == T - 1


@pytest.mark.parametrize("c,r,ps", [(24, 8, 4), (40, 6, 16), (128, 64, 16), (512, 2, 8)])
def test_gathered_contexts(c, r, ps):
    g = torch.Generator().manual_seed(c)
    lens = [5, 37, 1, 64]
    pool = torch.randn(40, 1, ps, c + r, generator=g).to(BF)
    order = torch.randperm(40, generator=g).tolist()
    tables = [[order.pop() for _ in range(-(-L // ps))] for L in lens]
    want = torch.cat([pool[tables[b][t // ps], 0, t % ps][None] for b, L in enumerate(lens) for t in range(L)])
    tables = [t + [-1] * (20 - len(t)) for t in tables]
    total = sum(lens)
    lat, rot = F().latent_gather(pool.to(DEV), i32(tables), i32(lens), total + 9, c, r)
    assert torch.equal(lat[:total].cpu(), want[:, :c]) and torch.equal(rot[:total, :r].cpu(), want[:, c:])
    assert rot.shape[1] == -(-r // 8) * 8
    assert float(lat[total:].float().abs().sum()) == 0.0 and float(rot[total:].float().abs().sum()) == 0.0


UNFOLDED = [(2, 8, 2, 8), (5, 24, 8, 40), (4, 64, 64, 64), (3, 128, 64, 128), (2, 136, 40, 96), (6, 72, 16, 48), (1, 192, 24, 72),
            (3, 64, 128, 64), (2, 64, 16, 128)]


@pytest.mark.parametrize("H,d,r,e", UNFOLDED)
@pytest.mark.parametrize("window", [0, 70])
def test_unfolded_prompt_attention(H, d, r, e, window):
    """Whole prompts, portions that start late and single tokens, unequal requests in one call, with and without a gate;
    rows of the output that belong to no request of the call stay as they are."""
    g = torch.Generator().manual_seed(d + e)
    lens, new, lead = [300, 129, 1, 70], [300, 40, 1, 2], 2
    assert F().prefill_attention_tc_unfolded_supported(d, r, e)
    cols, at = F().unfolded_query_layout(d, r)
    T = lead + sum(new)
    total = sum(lens)
    kv = torch.randn(total + 5, H * (d + e), generator=g).to(BF)
    kr = torch.randn(total + 5, -(-r // 8) * 8, generator=g).to(BF)
    q = torch.zeros(T, H, cols)
    q[..., :d], q[..., at:at + r] = torch.randn(T, H, d, generator=g), torch.randn(T, H, r, generator=g)
    q = q.to(BF)
    gate = torch.randn(T, 7 + H * e, generator=g)
    scale = (d + r) ** -0.5
    starts = [lead]
    for n in new:
        starts.append(starts[-1] + n)
    want, base = torch.zeros(T, H * e, dtype=torch.float64), 0
    for b, (L, n) in enumerate(zip(lens, new)):
        rows = slice(base, base + L)
        k = torch.cat([kv[rows, :H * d].double().view(L, H, d), kr[rows, :r].double()[:, None].expand(L, H, r)], -1)
        v = kv[rows, H * d:].double().view(L, H, e)
        qq = torch.cat([q[starts[b]:starts[b + 1], :, :d], q[starts[b]:starts[b + 1], :, at:at + r]], -1).double()
        i, j = torch.arange(L - n, L)[:, None], torch.arange(L)[None, :]
        mask = (j <= i) & ((i - j < window) if window else torch.ones(n, L, dtype=torch.bool))
        s = (torch.einsum("thd,jhd->htj", qq, k) * scale).masked_fill(~mask, float("-inf"))
        want[starts[b]:starts[b + 1]] = torch.einsum("htj,jhe->the", torch.softmax(s, -1), v).reshape(n, H * e)
        base += L
    for use_gate in (False, True):
        out = torch.full((T, H * e), 9.0, dtype=BF, device=DEV)
        F().prefill_attention_tc_unfolded(q.to(DEV), kv.to(DEV), kr.to(DEV), i32(starts), i32(lens), max(new), d, r, e,
                                          window, scale, out, gate.to(DEV) if use_gate else None, 7)
        F().check_tc_status()
        ref = want * torch.sigmoid(gate.double()[:, 7:]) if use_gate else want
        close(out[lead:], ref[lead:], 1.5e-2, f"gate {use_gate}")
        assert bool((out[:lead] == 9.0).all())


def test_a_far_key_in_the_unfolded_prompt_attention():
    """A key that stands out, hundreds of tokens back, at tile edges, and the query's own; the next key is not seen."""
    H, d, r, e, L = 2, 64, 16, 64, 700
    cols, at = F().unfolded_query_layout(d, r)
    g = torch.Generator().manual_seed(0)
    for part in ("plain", "rotated"):
        for key in (0, 63, 64, 127, 640, 698, 699):
            kv, kr = torch.randn(L, H * (d + e), generator=g) * 0.05, torch.randn(L, r, generator=g) * 0.05
            kv[:, 0:H * d:d] = 0.0
            kr[:, 0] = 0.0
            if part == "plain":
                kv[key, 0:H * d:d] = 6.0
            else:
                kr[key, 0] = 6.0
            kv[key, H * d:] = 3.0
            q = torch.zeros(L, H, cols)
            q[:, :, 0 if part == "plain" else at] = 6.0
            out = torch.zeros(L, H * e, dtype=BF, device=DEV)
            F().prefill_attention_tc_unfolded(q.to(BF).to(DEV), kv.to(BF).to(DEV), kr.to(BF).to(DEV), i32([0, L]), i32([L]),
                                              L, d, r, e, 0, 1.0, out)
            got = out.float().cpu()
            assert float((got[key:] - 3.0).abs().max()) < 0.05, (part, key)
            if key:
                assert float(got[:key].abs().max()) < 0.5, (part, key)
