"""The mechanisms of the Dinatar decoder one by one, each kernel against the formula written out in float64: linear attention
with a decay per key channel token by token and in chunks, over steps and shuffled slots, with decays of nought; attention with
falling scores and kept first positions through every kernel, with NaN in all that may not be read; sums of normed terms with a
layer norm behind them, embedding with position vectors, the router with a softmax over the chosen logits; and one key made to
stand out at every edge of a window and of the kept positions."""
import math

import pytest
import torch

from dinatar_helpers import config, gla, hgrn2, layer, left, lively_tensors, par, plain, plain_logits, rel_err, right, write_model

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
NAN = float("nan")


def ops():
    from beglin_b200.csrc import ops as o
    return o


def dev(t):
    return t.to(DEV).contiguous()


# ---------------------------------------------------------------------------------------------- linear attention
class Linear:
    """One way of making q, k, a, v from random rows, in float64 and as arguments of the kernels."""

    def __init__(self, forget, H, n, nv, seed, rank=5, tau=3.0, gate=True):
        g = self.g = torch.Generator().manual_seed(seed)
        self.forget, self.H, self.n, self.nv, self.rank, self.tau, self.gate = forget, H, n, nv, rank, tau, gate and not forget
        self.bias = 1.5 * torch.randn(H * n, generator=g)
        self.lower = 0.9 * torch.rand(H * n, generator=g) * (torch.rand(H * n, generator=g) < 0.6)
        self.wa = torch.randn(H * n, rank, generator=g)
        self.norm = 1.0 + 0.2 * torch.randn(nv, generator=g)
        self.pad = 3                                    # columns in front that nobody may read
        self.cols = {"q": self.pad, "k": self.pad + H * n, "v": self.pad + 2 * H * n, "g": self.pad + 2 * H * n + H * nv}
        self.cols["r"] = self.cols["g"] + (H * nv if self.gate else 0)
        self.width = self.cols["r"] + (0 if forget else rank)

    def rows(self, T):
        t = torch.randn(T, self.width, generator=self.g)
        t[:, :self.pad] = NAN
        return t

    def decode(self, rows):
        """(q, k, a, v, gate) in float64, [T, H, n] and [T, H, nv]."""
        r = rows.double()
        part = lambda name, m: r[:, self.cols[name]:self.cols[name] + self.H * m].reshape(-1, self.H, m)
        q, k, v = part("q", self.n), part("k", self.n), part("v", self.nv)
        shape = k.shape
        if self.forget:
            a = plain.forget_gate(k.reshape(-1, self.H * self.n) + self.bias.double(), self.lower.double()).view(shape)
            return plain.silu(q), 1.0 - a, a, v, None
        z = r[:, self.cols["r"]:self.cols["r"] + self.rank] @ self.wa.double().T + self.bias.double()
        return q * 0.7, k, plain.rooted_decay(z, self.tau).view(shape), v, part("g", self.nv) if self.gate else None

    def want(self, rows, state, eps=1e-5):
        q, k, a, v, gate = self.decode(rows)
        o, state = plain.decayed_readout(q, k, a, v, state)
        o = plain.rms_unit(o, eps) * self.norm.double()
        if gate is not None:
            o = o * plain.silu(gate)
        return o.reshape(rows.shape[0], -1), state

    def run(self, rows, state, slots, out, reqs=None, chunks=None, longs=None, eps=1e-5):
        kw = dict(lower=dev(self.lower), q_silu=True) if self.forget else \
            dict(decay_matrix=dev(self.wa), r_col=self.cols["r"], power=1.0 / self.tau, q_scale=0.7)
        count = lambda t: 0 if t is None else t.shape[0]
        ops().gated_linear_attention(dev(rows), self.cols["q"], self.cols["k"], self.cols["v"], dev(self.bias), dev(self.norm), eps, state,
                                     slots, reqs, count(reqs), out, self.H, self.n, self.nv, g_col=self.cols["g"] if self.gate else -1,
                                     chunks=chunks, n_chunks=count(chunks), longs=longs, n_long=count(longs), **kw)


@pytest.mark.parametrize("H,n,nv", [(1, 1, 1), (3, 10, 7), (2, 64, 64), (2, 48, 130), (2, 128, 128), (1, 5, 33), (1, 200, 24), (1, 16, 530)])
@pytest.mark.parametrize("forget", [True, False])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_linear_attention_token_by_token_in_chunks_over_steps_and_slots(H, n, nv, forget, dtype):
    """Three steps over four requests in shuffled slots with NaN in everything unwritten: portions of 1 to 200 rows, the long
    ones in chunks where the sizes allow it (heads of 16 x 530 walk with the state in memory), against the recurrence token by
    token."""
    from beglin_b200.engine.batch import cut_long_requests
    L = Linear(forget, H, n, nv, seed=H * 100 + n + nv)
    sz = H * n * nv
    state = torch.full((6, sz + 4), NAN, device=DEV)
    slot_of = [4, 0, 5, 2]
    state[slot_of, :sz] = 0.0
    slots = torch.tensor(slot_of, dtype=torch.int32, device=DEV)
    S = [None] * 4
    chunk = ops().gla_chunk(n, nv)
    assert bool(chunk) == (nv < 500)
    for lens in ([200, 1, 64, 3], [1, 70, 1, 129], [63, 17, 1, 16]):
        starts = [sum(lens[:i]) for i in range(4)]
        rows = L.rows(sum(lens))
        want = torch.zeros(sum(lens), H * nv, dtype=torch.float64)
        for i in range(4):
            sl = slice(starts[i], starts[i] + lens[i])
            want[sl], S[i] = L.want(rows[sl], S[i])
        short, chunks, longs = cut_long_requests(starts, lens, chunk or 64, 16 if chunk else 1 << 30)
        up = lambda a: torch.from_numpy(a).to(DEV)
        out = torch.full((sum(lens), H * nv), NAN, device=DEV, dtype=dtype)
        L.run(rows, state, slots, out, reqs=up(short) if len(short) else None, chunks=up(chunks) if len(chunks) else None,
              longs=up(longs) if len(longs) else None)
        for i in range(4):
            sl = slice(starts[i], starts[i] + lens[i])
            assert rel_err(out[sl], want[sl]) < (2e-5 if dtype == torch.float32 else 6e-3), (lens, i)
            assert rel_err(state[slot_of[i], :sz].view(H, n, nv), S[i]) < 5e-6, (lens, i)
    assert torch.isnan(state[[1, 3]]).all() and torch.isnan(state[:, sz:]).all()


def test_decays_of_nought_and_of_nearly_one():
    """A channel whose forget gate shuts altogether now and then (a decay of exactly nought beside decays close to one: a
    quotient of running products would be 0/0) and one that keeps a token over 900 rows; in chunks and row by row."""
    T, n, nv = 901, 2, 3
    L = Linear(True, 1, n, nv, seed=4)
    L.bias = torch.zeros(n)
    L.lower = torch.zeros(n)
    rows = L.rows(T)
    rows[:, L.cols["q"]:L.cols["q"] + n] = 1.0
    rows[:, L.cols["k"]] = 5.0
    rows[::37, L.cols["k"]] = -200.0                   # sigmoid(-200) is nought in float
    rows[:, L.cols["k"] + 1] = 9.0
    rows[0, L.cols["k"] + 1] = -9.0                    # the second channel writes the first token, and keeps most of it
    rows[0, L.cols["v"]:L.cols["v"] + nv] = torch.tensor([40.0, -20.0, 10.0])
    want, S = L.want(rows, None)
    for way in ("chunks", "rows"):
        state = torch.zeros(1, n * nv, device=DEV)
        out = torch.empty(T, nv, device=DEV)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
        if way == "rows":
            L.run(rows, state, i32([0]), out, reqs=i32([[0, 0, T]]))
        else:
            chunks = [[0, f, min(64, T - f), 0] for f in range(0, T, 64)]
            L.run(rows, state, i32([0]), out, chunks=i32(chunks), longs=i32([[0, 0, T, 0]]))
        assert torch.isfinite(out).all() and rel_err(out, want) < 2e-4, way          # (900 products of decays, each rounded)
        assert rel_err(state.view(1, n, nv), S) < 2e-4
    assert float(S[0, 1].abs().max()) > 20.0


# ---------------------------------------------------------------------------------------------- Mamba-2
@pytest.mark.parametrize("H,P,N,G", [(1, 4, 4, 1), (6, 36, 20, 2), (2, 128, 128, 1), (4, 64, 64, 4), (3, 100, 200, 1), (2, 7, 9, 1)])
@pytest.mark.parametrize("wdtype", [torch.float32, torch.bfloat16])
def test_mamba2_in_chunks_and_row_by_row_over_steps_and_slots(H, P, N, G, wdtype):
    """Three steps over four requests in shuffled slots with NaN in everything unwritten, portions of 64 rows and more in chunks
    where the sizes allow it (multiples of 4): step sizes from nearly nought to ones that forget everything, against the
    recurrence token by token."""
    from beglin_b200.engine.batch import cut_long_requests
    o = ops()
    g = torch.Generator().manual_seed(H * P + N)
    r = lambda *s: torch.randn(*s, generator=g)
    A_log, dt_bias, D = (r(H) * 1.5).to(wdtype), r(H).to(wdtype), r(H).to(wdtype)
    sz, width = H * N * P, H * P + 2 * G * N
    state = torch.full((6, sz + 4), NAN, device=DEV)
    slot_of = [4, 0, 5, 2]
    state[slot_of, :sz] = 0.0
    S = [torch.zeros(H, N, P, dtype=torch.float64) for _ in range(4)]
    chunk = o.ssm_chunk(H, P, N, G)
    assert bool(chunk) == (P % 4 == 0 and N % 4 == 0)
    for lens in ([200, 1, 64, 3], [1, 70, 1, 129], [65, 17, 1, 63]):
        T = sum(lens)
        starts = [sum(lens[:i]) for i in range(4)]
        xbc, raw = r(T, width), 3.0 * r(T, H + 2) - 2.0
        raw[::13] = 60.0                                   # a step that forgets the state, between small ones
        x, B, C = xbc[:, :H * P].double().view(T, H, P), xbc[:, H * P:H * P + G * N].double().view(T, G, N), xbc[:, H * P + G * N:].double().view(T, G, N)
        dt = torch.nn.functional.softplus(raw[:, 2:].double() + dt_bias.double())
        want = torch.zeros(T, H, P, dtype=torch.float64)
        for i in range(4):
            for t in range(starts[i], starts[i] + lens[i]):
                for h in range(H):
                    gg = h // (H // G)
                    S[i][h] = torch.exp(-torch.exp(A_log[h].double()) * dt[t, h]) * S[i][h] + dt[t, h] * torch.outer(B[t, gg], x[t, h])
                    want[t, h] = S[i][h].T @ C[t, gg] + D[h].double() * x[t, h]
        short, chunks, longs = cut_long_requests(starts, lens, chunk or 64, 64 if chunk else 1 << 30)
        up = lambda a: torch.from_numpy(a).to(DEV)
        y = torch.full((T, H * P), NAN, device=DEV)
        o.ssm_scan(dev(xbc), dev(raw), 2, dev(dt_bias), dev(A_log), dev(D), state, torch.tensor(slot_of, dtype=torch.int32, device=DEV),
                   up(short), len(short), y, H, P, N, G, up(chunks), len(chunks), up(longs), len(longs))
        for i in range(4):
            sl = slice(starts[i], starts[i] + lens[i])
            assert rel_err(y.view(T, H, P)[sl], want[sl]) < 5e-6, (lens, i)
            assert rel_err(state[slot_of[i], :sz].view(H, P, N).transpose(1, 2), S[i]) < 5e-6, (lens, i)
    assert torch.isnan(state[[1, 3]]).all() and torch.isnan(state[:, sz:]).all()


# ---------------------------------------------------------------------------------------------- attention
def paged(k, v, page, window, keep, first_query, dtype):
    """Keys [S, G, hd] and values [S, G, vd] of one request in shuffled pages; pages wholly in front of the first query's window
    and behind the kept positions are not held.  NaN wherever nothing was written."""
    S, G, hd = k.shape
    vd = v.shape[2]
    n_pages = -(-S // page)
    lo = max(0, first_query - window + 1) if window else 0
    held = [i for i in range(n_pages) if (i + 1) * page > lo or i * page < keep]
    order = torch.randperm(n_pages + 2, generator=torch.Generator().manual_seed(S)).tolist()
    flat = torch.full((n_pages + 2, G * page * (hd + vd)), NAN)
    table = torch.full((1, n_pages + 3), -1, dtype=torch.int32)
    for i in held:
        table[0, i] = order[i]
        kk, vv = torch.full((G, page, hd), NAN), torch.full((G, page, vd), NAN)
        m = min(page, S - i * page)
        kk[:, :m], vv[:, :m] = k[i * page:i * page + m].transpose(0, 1), v[i * page:i * page + m].transpose(0, 1)
        flat[order[i]] = torch.cat([kk.reshape(-1), vv.reshape(-1)])
    pool = flat if hd != vd else flat.view(n_pages + 2, 2, G, page, hd)
    return pool.to(dtype).to(DEV).contiguous(), table.to(DEV)


CASES = [  # kernel, dtype, query heads, kv heads, hd, vd, page, window, keep, positions, queries
    ("generic", torch.float32, 6, 2, 10, 14, 8, 20, 3, 150, 40),
    ("generic", torch.float32, 3, 1, 9, 9, 16, 40, 70, 230, 100),
    ("generic", torch.float32, 2, 2, 64, 64, 64, 300, 6, 700, 1),
    ("generic", torch.float32, 4, 1, 24, 8, 16, 0, 0, 130, 130),
    ("generic", torch.bfloat16, 4, 2, 32, 16, 16, 33, 5, 200, 60),
    ("mma_rows", torch.bfloat16, 4, 2, 64, 64, 16, 33, 5, 300, 170),
    ("mma_rows", torch.bfloat16, 2, 1, 128, 128, 64, 100, 130, 500, 200),
    ("mma_rows", torch.bfloat16, 8, 1, 64, 64, 48, 70, 6, 400, 90),
    ("tc_rows", torch.bfloat16, 4, 2, 64, 64, 16, 33, 5, 300, 170),
    ("tc_rows", torch.bfloat16, 2, 1, 128, 128, 64, 100, 130, 500, 200),
    ("tc_rows", torch.bfloat16, 6, 1, 64, 64, 64, 72, 6, 1100, 900),
    ("tc_rows", torch.bfloat16, 8, 8, 128, 128, 8, 0, 0, 400, 400),
    ("mma_keys", torch.bfloat16, 4, 2, 64, 64, 16, 33, 5, 700, 1),
    ("mma_keys", torch.bfloat16, 2, 1, 128, 128, 64, 300, 130, 1500, 1),
    ("mma_keys", torch.bfloat16, 24, 2, 64, 64, 64, 40, 7, 2500, 1),
    ("mma_keys", torch.bfloat16, 8, 1, 64, 64, 48, 600, 6, 900, 1),
    ("mma_keys", torch.bfloat16, 6, 2, 64, 64, 64, 72, 300, 1300, 1),
    ("mma_keys", torch.bfloat16, 4, 4, 64, 64, 32, 0, 0, 600, 1),
]


@pytest.mark.parametrize("case", CASES, ids=[f"{c[0]}-{c[7]}-{c[8]}-{c[9]}-{c[4]}" for c in CASES])
def test_falling_scores_and_kept_positions(case):
    """Values and queries such that single keys carry the result (a window or a kept range one position off shows), every page
    that need not be held taken away."""
    kernel, dtype, H, G, hd, vd, page, window, keep, S, T = case
    g = torch.Generator().manual_seed(S + T)
    q, k, v = (torch.randn(*s, generator=g) for s in ((T, H, hd), (S, G, hd), (S, G, vd)))
    first = S - T
    # the keys at the edges stand out for every query: the oldest of the window, the one in front of it, the last kept, the next
    for p in {max(0, first - window + 1) if window else 0, max(0, first - window), keep - 1, keep, S - 1 - max(window - 1, 0)}:
        if 0 <= p < S:
            k[p] = 1.2 * q[0, 0] * math.sqrt(hd) / q[0, 0].norm()
    q = (0.4 * q + q[0, 0]).to(dtype)
    k, v = k.to(dtype), v.to(dtype)
    slopes = [plain.falling_slope(h, H) * 0.3 for h in range(H)]
    want = torch.cat([one_query(q[t], k, v, 0.11, first + t, window, keep, slopes) for t in range(T)])
    pool, table = paged(k.float(), v.float(), page, window, keep, first, dtype)
    o = ops()
    i32 = lambda a: torch.tensor(a, dtype=torch.int32, device=DEV)
    bq = {"generic": None, "mma_rows": 64 // (H // G), "tc_rows": 128 // (H // G), "mma_keys": 1}[kernel]
    tile = 64
    if kernel == "generic":
        _, bq, tile = o.attention_plan(H // G, hd, dtype, False, "generic", page, vd=vd)
    qblk = i32([[0, r, min(bq, T - r)] for r in range(0, T, bq)])
    out = torch.full((T, H * vd), NAN, dtype=dtype, device=DEV)
    status = o.new_status(DEV)
    qd = dev(q.view(T, H * hd))
    o.attention(qd, qd.stride(0), pool, table, i32(list(range(first, S))), qblk, qblk.shape[0], S - 1, T, H, G, hd, window, 64, tile, bq,
                0.11, out, status, kernel, vd=vd, keep=keep if window else 0, slopes=dev(torch.tensor(slopes)))
    o.raise_on_status(status)
    assert torch.isfinite(out.float()).all()
    assert rel_err(out.view(T, H, vd), want) < (1e-5 if dtype == torch.float32 else 1.2e-2)


def one_query(q, k, v, scale, pos, window, keep, slopes):
    """[1, H, vd]: one query at position `pos` over keys [S, G, hd]."""
    H, G = q.shape[0], k.shape[1]
    keys = plain.visible(pos, window or None, keep)
    back = torch.tensor([float(pos - j) for j in keys], dtype=torch.float64)
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (k[keys, g].double() @ q[h].double()) * scale - slopes[h] * back
        out.append(torch.softmax(s, -1) @ v[keys, g].double())
    return torch.stack(out)[None]


# ---------------------------------------------------------------------------------------------- around the stream
@pytest.mark.parametrize("T,d", [(3, 40), (70, 256), (2, 75), (600, 1030), (1, 1031), (520, 64)])
def test_sum_of_normed_terms_and_the_layer_norm_behind_it(T, d):
    from beglin_b200.parts.stream import NormedTerm
    g = torch.Generator().manual_seed(d)
    r = lambda *s: torch.randn(*s, generator=g)
    x, a, b, c = r(T, d), 3.0 * r(T, d).to(torch.bfloat16), 0.2 * r(3, T, d), r(T, d)
    wa, wb, w, s = 1 + 0.3 * r(d), 1 + 0.3 * r(d), 1 + 0.2 * r(d), 0.4 * r(d)
    x += 5.0                                           # a mean worth taking off
    want = x.double() + 0.5 * plain.rms_unit(a.double(), 1e-3) * wa.double() + 0.5 * plain.rms_unit(b.double().sum(0), 1e-3) * wb.double() \
        - 2.0 * c.double()
    for dt in (torch.float32, torch.bfloat16):
        xs, h = dev(x.clone()), torch.empty(T, d, device=DEV, dtype=dt)
        terms = [(NormedTerm(dev(a), dev(wa), 1e-3), 0.5), (NormedTerm(dev(b), dev(wb), 1e-3), 0.5), (dev(c), -2.0)]
        ops().add_terms_norm(xs, terms, weight1=dev(w), bias1=dev(s), eps=1e-4, out1=h, center=True)
        assert rel_err(xs, want) < 1e-6
        assert rel_err(h, plain.layer_norm(want, w.double(), s.double(), 1e-4)) < (2e-6 if dt == torch.float32 else 5e-3)
        assert rel_err(terms[0][0].float().cpu(), plain.rms_unit(a.double(), 1e-3) * wa.double()) < 1e-6
    # the same norm where nothing is owed, at some rows only
    rows = torch.tensor([T - 1, 0], dtype=torch.int32, device=DEV)
    h = torch.empty(2, d, device=DEV)
    ops().add_layernorm(dev(x), None, dev(w), 1e-4, h, rows=rows, update=False, bias=dev(s))
    assert rel_err(h, plain.layer_norm(x.double(), w.double(), s.double(), 1e-4)[[T - 1, 0]]) < 2e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_embedded_rows_with_position_vectors(dtype):
    g = torch.Generator().manual_seed(1)
    table, pos = torch.randn(9, 37, generator=g).to(dtype), torch.randn(6, 37, generator=g).to(dtype)
    i32 = lambda a: torch.tensor(a, dtype=torch.int32, device=DEV)
    out, status = torch.empty(4, 37, device=DEV), ops().new_status(DEV)
    ops().embed_gather(dev(table), i32([8, 0, 3, 3]), out, status, scale=2.5, pos_table=dev(pos), positions=i32([5, 0, 1, 4]))
    ops().raise_on_status(status)
    assert rel_err(out, 2.5 * table.double()[[8, 0, 3, 3]] + pos.double()[[5, 0, 1, 4]]) < 1e-6
    ops().embed_gather(dev(table), i32([8, 0, 3, 3]), out, status, scale=2.5, pos_table=dev(pos), positions=i32([5, 0, 6, 4]))
    with pytest.raises(ops().KernelError, match="position"):
        ops().raise_on_status(status)


@pytest.mark.parametrize("T,d,E,top", [(1, 8, 1, 1), (7, 24, 5, 2), (300, 64, 20, 4), (19, 33, 9, 9)])
def test_router_with_a_bias_on_the_logits_and_a_softmax_over_the_chosen(T, d, E, top):
    g = torch.Generator().manual_seed(T + E)
    h = torch.randn(T, d, generator=g)
    W, bias = torch.randn(E, d, generator=g) * 6.0 / math.sqrt(d), 3.0 * torch.randn(E, generator=g)
    z = h.double() @ W.double().T + bias.double()
    ids, w = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    for from_logits in (False, True):
        if from_logits:
            ops().route_topk(dev((h.double() @ W.double().T).float()), top, ids, w, sigmoid="softmax_chosen", logit_bias=dev(bias))
        else:
            ops().route(dev(h), dev(W), top, ids, w, sigmoid="softmax_chosen", logit_bias=dev(bias))
        for t in range(T):
            order = sorted(range(E), key=lambda e: (-float(z[t, e]), e))[:top]
            assert ids[t].tolist() == order, t
            assert rel_err(w[t], torch.softmax(z[t, order], -1)) < 2e-5
    with pytest.raises(ops().KernelError, match="no choice bias"):
        ops().route(dev(h), dev(W), top, ids, w, sigmoid="softmax_chosen", bias=dev(bias))


@pytest.mark.parametrize("rows,n", [(3, 7), (5, 64), (130, 200)])
def test_square_of_relu(rows, n):
    g = torch.Generator().manual_seed(n)
    z = torch.randn(2, rows, n, generator=g)
    for dt in (torch.float32, torch.bfloat16):
        out = torch.empty(rows, n, device=DEV, dtype=dt)
        ops().activation(dev(z), out, "relu2")
        assert rel_err(out, plain.relu_squared(z.double().sum(0))) < (1e-6 if dt == torch.float32 else 5e-3)


# ---------------------------------------------------------------------------------------------- one key that stands out
SIZE, KEEP = 37, 6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hd,vd,page", [(64, 64, 16), (40, 24, 8)])
def test_a_key_that_stands_out_at_every_edge(tmp_path, dtype, hd, vd, page):
    """A model of ONE layer of two branches in which token 1 has a key that every query points along, under a scale that lets it
    carry the softmax wherever it is seen.  It stands on the last kept position, right behind it, and further on, so that
    queries see it just inside the window and just outside, in prompts and in single tokens: the logits are those of the plain
    implementation, and the plain implementation itself says that an edge one position off gives other logits."""
    d, vocab = 32, 12
    cfg = config(vocab, d, 1e-6, [layer(par(left(2, 1, hd, vd, 0.5, window=SIZE, keep=KEEP), right(1, 8, 4, 1, 2, 1)))], max_positions=256)
    t = lively_tensors(cfg, 1, torch.float32)
    g = torch.Generator().manual_seed(3)
    small = lambda name: torch.randn(t[name].shape, generator=g) * 0.02
    t["embed"] = torch.randn(vocab, d, generator=g) * 0.3
    t["embed"][1] = 0.0
    t["embed"][:, 0] = 0.0
    t["embed"][1, 0] = 6.0
    t["embed"][:, 1] = 3.0                                 # every token's
    t["pos"] = torch.zeros_like(t["pos"])
    t["l0.norm1"], t["l0.norm1.b"] = torch.ones(d), torch.zeros(d)
    t["l0.mix.left.out"] = torch.full((d,), 8.0)           # the attention's branch outweighs the embedded row in the logits
    m = "l0.mix.left."
    for name in ("q", "k", "q.b", "k.b"):
        t[m + name] = small(m + name)
    t[m + "k"][20, :2] = torch.tensor([3.0, 0.0])          # a key's feature 20 is the row's feature 0: token 1 alone
    t[m + "q.b"][[20, hd + 20]] = 8.0                      # a query's feature 20 is a constant
    stored = torch.float32 if dtype == "float32" else torch.bfloat16
    folder = write_model(str(tmp_path / "m"), cfg, {k: v.to(stored) for k, v in t.items()})
    # the last kept position (seen for good: nothing further on may stand out beside it), the first that is not, and further on
    for marks, changes in (((5,), [("keep_first", KEEP - 1)]), ((6, 74), [("keep_first", KEEP + 1), ("size", SIZE - 1), ("size", SIZE + 1)]),
                           ((60, 111), [("size", SIZE - 1), ("size", SIZE + 1)])):
        ids = [2 + (i * 7) % 10 for i in range(130)]
        for p in marks:
            ids[p] = 1
        want = plain_logits(folder, ids)
        from beglin_b200 import Engine
        import replay_lib as rl
        for way in ("whole", "cut"):
            eng = Engine.from_folder(folder, dtype=dtype, max_tokens=192, page_size=page, max_requests=2, kv_split=64)
            if way == "whole":
                steps = [{"entries": [{"id": "a", "tokens": ids, "want": list(range(130))}], "end": ["a"]}]
            else:
                steps = [{"entries": [{"id": "a", "tokens": ids[:35], "want": list(range(35))}]},
                         {"entries": [{"id": "a", "tokens": ids[35:90], "want": list(range(55))}]}]
                steps += [{"entries": [{"id": "a", "tokens": [ids[i]], "want": [0]}], "end": ["a"] if i == 129 else []}
                          for i in range(90, 130)]
            got = rl.run_in_process(eng, steps)
            rows = torch.stack([got[("a", p)] for p in range(130)])
            assert rel_err(rows, want) < (3e-5 if dtype == "float32" else 4e-2), (way, marks)
        cfg_w, w = plain.read_folder(folder, torch.float64)
        mask = cfg_w["layers"][0]["mixer"]["left"]["mask"]
        for key, value in changes:
            old, mask[key] = mask[key], value
            assert rel_err(plain.forward(cfg_w, w, ids), want) > 0.2, (key, value, marks)
            mask[key] = old


@pytest.mark.parametrize("kind", ["hgrn2", "gla"])
def test_a_token_far_back_is_still_in_the_state(tmp_path, kind):
    """A model of ONE layer of linear attention whose decays keep what token 1 writes: 300 positions on it still decides the
    result, through chunks of a prompt and single tokens; the plain implementation with another token in its place gives other
    logits."""
    d, vocab, n = 24, 10, 300
    cfg = config(vocab, d, 1e-6, [layer(hgrn2(1, 8, 8) if kind == "hgrn2" else gla(1, 8, 8, 16.0, 4))], max_positions=512)
    t = lively_tensors(cfg, 5, torch.float32)
    t["pos"] *= 0.0
    if kind == "hgrn2":
        t["l0.mix.lower"][:] = 0.9995
    else:
        t["l0.mix.a2.b"][:] = 7.0
        t["l0.mix.a2"] *= 0.1
    t["embed"][:, 0] = 0.0                                      # rows of mean nought, in which feature 0 is token 1's alone
    t["embed"][:, 1:] -= t["embed"][:, 1:].mean(1, keepdim=True)
    t["embed"][1] = -12.0 / (d - 1)
    t["embed"][1, 0] = 12.0
    t["l0.norm1"] = torch.ones(d)
    t["l0.norm1.b"] = torch.zeros(d)
    t["l0.mix.v"] *= 0.05
    t["l0.mix.v"][:, 0] = torch.linspace(-9.0, 9.0, 8)         # the values are large where a row's feature 0 is: token 1 alone
    folder = write_model(str(tmp_path / "m"), cfg, t)
    ids = [2 + (i * 3) % 8 for i in range(n)]
    ids[7] = 1
    other = list(ids)
    other[7] = 3
    want = plain_logits(folder, ids)
    assert rel_err(plain_logits(folder, other)[-1], want[-1]) > 0.1
    from beglin_b200 import Engine
    eng = Engine.from_folder(folder, dtype="float32", max_tokens=512, page_size=16, max_requests=2)
    rows = eng.step([("a", ids[:270], [269])])
    assert rel_err(rows[0], want[269]) < 1e-4
    for i in range(270, n):
        rows = eng.step([("a", [ids[i]], [0])])
        assert rel_err(rows[0], want[i]) < 1e-4
