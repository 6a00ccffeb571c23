"""The mechanisms of the Fanitar decoder one by one, each kernel against the formula written out in float64: rotation and append of
heads made of two maps, differential attention through every kernel with NaN in all that may not be read, keys made to stand out for
one map at the borders of tiles, pages and ranges; the step between two sublayers with norms in front and behind; the clamped gate in
every product that has it; latent attention with a sink and a gate per feature at a window's edges."""
import math

import pytest
import torch

from fanitar_helpers import config, dense, lat, layer, lively_tensors, plain, plain_logits, rel_err, write_model

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
NAN = float("nan")


def ops():
    from beglin_b200.csrc import ops as o
    return o


def dev(t):
    return t.to(DEV).contiguous()


def i32(a):
    return torch.tensor(a, dtype=torch.int32, device=DEV)


# ---------------------------------------------------------------------------------------------- rotation and append
APPEND = [  # query heads, kv heads, dim, vdim, rotated, interleaved, stored map, stored value, page
    (3, 1, 10, 7, 6, False, 10, 7, 4),
    (4, 2, 5, 13, 0, False, 5, 13, 8),
    (2, 2, 12, 24, 12, True, 32, 64, 16),
    (4, 1, 40, 88, 32, False, 64, 128, 16),
    (6, 2, 64, 128, 32, False, 64, 128, 64),
    (2, 1, 24, 40, 16, True, 32, 64, 8),
    (12, 2, 64, 128, 64, False, 64, 128, 64),
]


@pytest.mark.parametrize("case", APPEND, ids=["-".join(map(str, c)) for c in APPEND])
@pytest.mark.parametrize("dtype,parts,padded", [(torch.float32, 1, False), (torch.bfloat16, 1, False), (torch.bfloat16, 3, True),
                                                (torch.float32, 2, True)])
def test_rotation_and_append_of_heads_made_of_two_maps(case, dtype, parts, padded):
    H, G, n, nv, rot, inter, kw, vw, page = case
    T = 11
    g = torch.Generator().manual_seed(n + nv)
    width = -(-(2 * n * (H + G) + nv * G) // 8) * 8 + 8                 # (columns behind that nobody may read)
    full = torch.randn(T, width, generator=g)
    full[:, 2 * n * (H + G) + nv * G:] = NAN
    src = full.to(dtype) if parts == 1 else torch.stack([full * 0.25] * (parts - 1) + [full * (1.0 - 0.25 * (parts - 1))]).contiguous()
    full = src.double() if parts == 1 else src.double().sum(0)
    pos = [5, 6, 7, 8, 9, 0, 1, 2, 30, 31, 3]                          # two requests' rows, the second one's out of order
    req = [0] * 5 + [1] * 6
    angle = torch.tensor(pos, dtype=torch.float64)[:, None] * (40.0 ** (-2.0 * torch.arange(max(rot // 2, 1), dtype=torch.float64) / max(rot, 2)))
    cs = torch.stack([torch.cos(angle), torch.sin(angle)], -1).float()

    def turn(x):                                                        # [T, heads, n]
        out = x.clone()
        for i in range(rot // 2):
            a, b = (2 * i, 2 * i + 1) if inter else (i, i + rot // 2)
            c, s = cs[:, i, 0].double()[:, None], cs[:, i, 1].double()[:, None]
            out[..., a], out[..., b] = x[..., a] * c - x[..., b] * s, x[..., b] * c + x[..., a] * s
        return out
    q = turn(full[:, :2 * n * H].reshape(T, 2 * H, n))
    k = turn(full[:, 2 * n * H:2 * n * (H + G)].reshape(T, 2 * G, n))
    v = full[:, 2 * n * (H + G):2 * n * (H + G) + nv * G].reshape(T, G, nv)
    n_pages = 32 // page + 1
    table = i32([[n_pages + i for i in range(n_pages)], list(range(n_pages))])
    pool = torch.full((2 * n_pages, G * page * (2 * kw + vw)), NAN, dtype=dtype, device=DEV)
    qw = 2 * kw if padded else kw
    qo = torch.full((T, 2 * H * qw), NAN, dtype=dtype, device=DEV)
    status = ops().new_status(DEV)
    ops().qk_norm_rope_append(dev(src), qo, T, 2 * H, G, n, nv, rot, inter, None, None, 0.0, dev(cs) if rot else None, i32(pos), i32(req),
                              table, pool, page, status, maps=2, stored=(kw, vw), padded=padded)
    ops().raise_on_status(status)
    tol = 1e-6 if dtype == torch.float32 else 5e-3
    got = qo.view(T, H, 2, qw).cpu().double()
    want = torch.zeros_like(got)
    for c in range(2):
        at = c * kw if padded else 0
        want[:, :, c, at:at + n] = q.view(T, H, 2, n)[:, :, c]
    assert rel_err(got, want) < tol
    keys = pool[:, :G * page * 2 * kw].view(2 * n_pages, G, page, 2, kw)
    values = pool[:, G * page * 2 * kw:].view(2 * n_pages, G, page, vw)
    written = torch.zeros(2 * n_pages, page, dtype=torch.bool)
    for t in range(T):
        pg, slot = int(table[req[t], pos[t] // page]), pos[t] % page
        written[pg, slot] = True
        kk, vv = torch.zeros(G, 2, kw, dtype=torch.float64), torch.zeros(G, vw, dtype=torch.float64)
        kk[:, :, :n], vv[:, :nv] = k[t].view(G, 2, n), v[t]
        assert rel_err(keys[pg, :, slot], kk) < tol and rel_err(values[pg, :, slot], vv) < tol
    assert torch.isnan(keys.cpu()[~written[:, None, :].expand(-1, G, -1)].float()).all()


# ---------------------------------------------------------------------------------------------- differential attention
def paged(k, v, kw, vw, page, window, first_query, dtype):
    """Keys [S, G, 2, n] and values [S, G, nv] of one request in shuffled pages, features behind a map's or a value's own nought;
    pages wholly in front of the first query's window are not held.  NaN wherever nothing was written."""
    S, G, _, n = k.shape
    nv = v.shape[2]
    n_pages = -(-S // page)
    lo = max(0, first_query - window + 1) if window else 0
    order = torch.randperm(n_pages + 2, generator=torch.Generator().manual_seed(S)).tolist()
    flat = torch.full((n_pages + 2, G * page * (2 * kw + vw)), NAN)
    table = torch.full((1, n_pages + 3), -1, dtype=torch.int32)
    for i in range(n_pages):
        if (i + 1) * page <= lo:
            continue
        table[0, i] = order[i]
        kk, vv = torch.full((G, page, 2, kw), NAN), torch.full((G, page, vw), NAN)
        m = min(page, S - i * page)
        kk[:, :m], vv[:, :m] = 0.0, 0.0
        kk[:, :m, :, :n] = k[i * page:i * page + m].transpose(0, 1)
        vv[:, :m, :nv] = v[i * page:i * page + m].transpose(0, 1)
        flat[order[i]] = torch.cat([kk.reshape(-1), vv.reshape(-1)])
    pool = flat.view(n_pages + 2, 2, G, page, vw) if 2 * kw == vw else flat
    return pool.to(dtype).to(DEV).contiguous(), table.to(DEV)


def want_difference(q, k, v, scale, first, window, lam, out_scale, eps):
    """q [T, H, 2, n] at positions first .. first + T - 1 over k [S, G, 2, n], v [S, G, nv]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    q, k, v = q.double(), k.double(), v.double()
    out = torch.zeros(T, H, v.shape[2], dtype=torch.float64)
    for t in range(T):
        keys = plain.visible(first + t, window or None)
        for h in range(H):
            a = [torch.softmax((k[keys, h // (H // G), c] @ q[t, h, c]) * scale, -1) @ v[keys, h // (H // G)] for c in range(2)]
            out[t, h] = plain.rms_unit(a[0] - lam * a[1], eps) * out_scale
    return out


def run_difference(kernel, q, k, v, kw, vw, page, window, first, scale, lam, out_scale, eps, dtype, split=64):
    o = ops()
    T, H, _, n = q.shape
    S, G = k.shape[:2]
    nv = v.shape[2]
    pool, table = paged(k.float(), v.float(), kw, vw, page, window, first, dtype)
    planned, bq, tile = o.difference_plan(H // G, kw, vw, dtype, kernel == "mma_keys", "generic" if kernel == "generic" else "auto", page)
    assert planned == kernel
    padded = kernel == "mma_keys"
    rows = torch.zeros(T, H, 2, 2 * kw if padded else kw)
    for c in range(2):
        at = c * kw if padded else 0
        rows[:, :, c, at:at + n] = q[:, :, c].float()
    qblk = None if padded else i32([[0, r, min(bq, T - r)] for r in range(0, T, bq)])
    out = torch.full((T, H * nv), NAN, dtype=dtype, device=DEV)
    status = o.new_status(DEV)
    o.difference_attention(dev(rows.view(T, -1).to(dtype)), pool, table, i32(list(range(first, first + T))), qblk,
                           T if padded else qblk.shape[0], S - 1, T, H, G, kw, vw, nv, window, split, tile, bq, scale, lam, out_scale, eps,
                           out, status, kernel)
    o.raise_on_status(status)
    assert torch.isfinite(out.float()).all()
    return out.view(T, H, nv)


CASES = [  # kernel, dtype, query heads, kv heads, dim, vdim, stored map, stored value, page, window, positions, queries
    ("generic", torch.float32, 6, 2, 10, 14, 10, 14, 8, 20, 150, 40),
    ("generic", torch.float32, 3, 1, 9, 9, 9, 9, 16, 0, 230, 100),
    ("generic", torch.float32, 2, 2, 64, 128, 64, 128, 64, 300, 700, 1),
    ("generic", torch.float32, 4, 1, 130, 200, 130, 200, 16, 0, 130, 9),
    ("generic", torch.float32, 1, 1, 1, 1, 1, 1, 4, 0, 33, 33),
    ("generic", torch.bfloat16, 4, 2, 32, 16, 32, 16, 16, 33, 200, 60),
    ("generic", torch.bfloat16, 4, 1, 40, 88, 64, 128, 16, 0, 200, 60),
    ("tc_rows", torch.bfloat16, 4, 2, 32, 64, 32, 64, 16, 0, 300, 300),
    ("tc_rows", torch.bfloat16, 2, 1, 64, 128, 64, 128, 64, 0, 500, 200),
    ("tc_rows", torch.bfloat16, 6, 2, 40, 104, 64, 128, 16, 0, 140, 140),
    ("tc_rows", torch.bfloat16, 6, 1, 24, 40, 32, 64, 64, 72, 1100, 900),
    ("tc_rows", torch.bfloat16, 3, 3, 40, 21, 64, 128, 8, 0, 333, 70),
    ("tc_rows", torch.bfloat16, 1, 1, 64, 128, 64, 128, 32, 0, 63, 63),
    ("tc_rows", torch.bfloat16, 9, 3, 17, 64, 32, 64, 64, 0, 65, 2),
    ("tc_rows", torch.bfloat16, 5, 1, 64, 100, 64, 128, 4, 130, 420, 333),
    ("mma_keys", torch.bfloat16, 4, 2, 32, 64, 32, 64, 16, 0, 700, 1),
    ("mma_keys", torch.bfloat16, 2, 1, 64, 128, 64, 128, 64, 300, 1500, 1),
    ("mma_keys", torch.bfloat16, 16, 2, 56, 88, 64, 128, 64, 0, 2500, 1),
    ("mma_keys", torch.bfloat16, 4, 1, 24, 33, 32, 64, 48, 600, 900, 1),
    ("mma_keys", torch.bfloat16, 4, 4, 64, 128, 64, 128, 32, 0, 1, 1),
]


@pytest.mark.parametrize("case", CASES, ids=[f"{c[0]}-{'-'.join(map(str, c[2:]))}" for c in CASES])
def test_differential_attention(case):
    """The two maps of a head draw their weights from keys that stand out for one of them only, so that maps changed over, a map
    that reads the other's keys, or a window one position off shows; the difference weight lies close to one, where the two maps'
    results cancel where they agree."""
    kernel, dtype, H, G, n, nv, kw, vw, page, window, S, T = case
    g = torch.Generator().manual_seed(S + T + n)
    q, k, v = (torch.randn(*s, generator=g) for s in ((T, H, 2, n), (S, G, 2, n), (S, G, nv)))
    first = S - T
    for j, p in enumerate(sorted({max(0, first - window + 1) if window else 0, max(0, first - window), S - 1, S // 2, (S // 128) * 64})):
        c = j % 2
        k[p, :, c] = 1.3 * q[0, 0, c] * math.sqrt(n) / q[0, 0, c].norm()
    q = (0.4 * q + q[0, 0]).to(dtype)
    k, v = k.to(dtype), v.to(dtype)
    scale, lam, out_scale, eps = 1.4 / math.sqrt(n), 0.85, 0.4, 1e-5
    want = want_difference(q, k, v, scale, first, window, lam, out_scale, eps)
    got = run_difference(kernel, q, k, v, kw, vw, page, window, first, scale, lam, out_scale, eps, dtype)
    # (the norm magnifies the rounding of the weights where the maps nearly cancel: measured against each row's own condition)
    err = (got.double().cpu() - want).abs().amax(-1) / want.abs().amax(-1).clamp_min(1e-12)
    bound = 3e-5 if dtype == torch.float32 else 0.06
    assert float(err.median()) < bound / 3 and float((err > bound).double().mean()) <= 0.02, (float(err.max()), float(err.median()))


@pytest.mark.parametrize("kernel,dtype", [("generic", torch.float32), ("tc_rows", torch.bfloat16), ("mma_keys", torch.bfloat16)])
@pytest.mark.parametrize("map_", [0, 1])
def test_one_key_stands_out_for_one_map(kernel, dtype, map_):
    """One key after another at the borders of tiles, pages and ranges carries all the weight of one map, while the other map
    looks everywhere alike: the head's result is that key's value less the mean value (or the mean less lambda times it)."""
    S, n, nv = 400, 64, 128
    g = torch.Generator().manual_seed(3)
    v = torch.randn(S, 1, nv, generator=g).to(dtype)
    lam, out_scale, eps = 0.6, 0.7, 1e-6
    for p in (0, 1, 62, 63, 64, 65, 127, 128, 191, 192, 255, 256, 257, 319, 320, 398, 399):
        k = torch.zeros(S, 1, 2, n)
        k[p, 0, map_, 3] = 8.0
        q = torch.zeros(1, 1, 2, n)
        q[0, 0, map_, 3] = 6.0
        got = run_difference(kernel, q.to(dtype), k.to(dtype), v, 64, 128, 16, 0, S - 1, 1.0, lam, out_scale, eps, dtype)[0, 0]
        one, mean = v[p, 0].double(), v[:, 0].double().mean(0)
        o = one - lam * mean if map_ == 0 else mean - lam * one
        assert rel_err(got, plain.rms_unit(o, eps) * out_scale) < (1e-5 if dtype == torch.float32 else 2e-2), p


def test_rows_alone_and_together():
    """Portions of three requests and single tokens of two more in one launch of each kernel that takes portions, against every row
    alone (pages of all requests in one pool)."""
    o = ops()
    H, G, n, nv, kw, vw, page = 4, 2, 32, 64, 32, 64, 16
    g = torch.Generator().manual_seed(9)
    lens, starts = [70, 1, 33, 1, 2], [0, 129, 47, 64, 15]
    T = sum(lens)
    n_pages = 12
    pool = torch.randn(60, 2, G, page, vw, generator=g).to(torch.bfloat16)
    table = torch.randperm(60, generator=g)[:5 * n_pages].view(5, n_pages).int()
    q = torch.randn(T, H, 2, kw, generator=g).to(torch.bfloat16)
    rows0 = [sum(lens[:i]) for i in range(5)]
    pos = [s + j for s, l in zip(starts, lens) for j in range(l)]
    status = o.new_status(DEV)
    outs = {}
    for kernel, prefer in (("tc_rows", "auto"), ("generic", "generic")):
        _, bq, tile = o.difference_plan(H // G, kw, vw, torch.bfloat16, False, prefer, page)
        run = lambda blocks: (lambda out: (o.difference_attention(
            dev(q.view(T, -1)), dev(pool), dev(table), i32(pos), i32(blocks), len(blocks), max(pos), T, H, G, kw, vw, nv, 0, 64, tile, bq,
            0.2, 0.7, 0.5, 1e-5, out, status, kernel), out)[1])(torch.full((T, H * nv), NAN, dtype=torch.bfloat16, device=DEV))
        outs[kernel] = run([[i, rows0[i] + r, min(bq, lens[i] - r)] for i in range(5) for r in range(0, lens[i], bq)])
        for i in range(5):
            alone = run([[i, rows0[i] + r, min(bq, lens[i] - r)] for r in range(0, lens[i], bq)])
            sl = slice(rows0[i], rows0[i] + lens[i])
            assert torch.equal(alone[sl], outs[kernel][sl]), (kernel, i)
    o.raise_on_status(status)
    assert torch.isfinite(outs["tc_rows"].float()).all() and rel_err(outs["tc_rows"], outs["generic"]) < 2e-2


# ---------------------------------------------------------------------------------------------- between two sublayers
@pytest.mark.parametrize("T,d", [(3, 40), (70, 256), (2, 75), (600, 1030), (1, 1536), (9, 4096), (130, 5000), (2, 13000), (5, 17000)])
@pytest.mark.parametrize("weights", [torch.float32, torch.bfloat16])
def test_result_norm_sum_and_next_norm_in_one_pass(T, d, weights):
    """Every combination of what is owed (a result in either type or as partial sums, the embedded rows, a learned row) and of
    what is asked for (the new rows alone, or normed for the next sublayer)."""
    g = torch.Generator().manual_seed(d)
    r = lambda *s: torch.randn(*s, generator=g)
    x, e, vec = r(T, d), r(T, d), r(d)
    wy, w = (1 + 0.3 * r(d)).to(weights), (1 + 0.3 * r(d)).to(weights)
    for y in (None, r(T, d), 3.0 * r(T, d).to(torch.bfloat16), 0.2 * r(5, T, d)):
        for rows, vector in ((None, None), (e, vec), (None, vec)):
            if y is None and vector is None:
                continue
            want = x.double()
            if y is not None:
                want = want + plain.rms_norm(y.double().reshape(-1, T, d).sum(0), wy.double(), 1e-3)
            if rows is not None:
                want = want + rows.double()
            if vector is not None:
                want = want + vector.double()
            for out_type in (None, torch.float32, torch.bfloat16):
                xs = dev(x.clone())
                h = None if out_type is None else torch.full((T, d), NAN, device=DEV, dtype=out_type)
                ops().norm_step(xs, None if y is None else dev(y), None if y is None else dev(wy), 1e-3, rows=None if rows is None else dev(rows),
                                vector=None if vector is None else dev(vector), weight=None if h is None else dev(w), eps=1e-4, out=h)
                assert rel_err(xs, want) < 2e-6
                if h is not None:
                    assert rel_err(h, plain.rms_norm(want, w.double(), 1e-4)) < (3e-6 if out_type == torch.float32 else 5e-3)


def test_a_row_of_the_step_does_not_depend_on_the_others():
    g = torch.Generator().manual_seed(2)
    x, y, w = torch.randn(90, 1032, generator=g), torch.randn(90, 1032, generator=g), torch.ones(1032)
    run = lambda sl: (lambda xs, h: (ops().norm_step(xs, dev(y[sl]), dev(w), 1e-5, weight=dev(w), eps=1e-5, out=h), (xs.cpu(), h.cpu()))[1])(
        dev(x[sl].clone()), torch.empty(len(range(*sl.indices(90))), 1032, device=DEV))
    whole = run(slice(0, 90))
    for a, b in ((0, 1), (17, 19), (40, 90)):
        part = run(slice(a, b))
        assert torch.equal(part[0], whole[0][a:b]) and torch.equal(part[1], whole[1][a:b])


# ---------------------------------------------------------------------------------------------- the clamped gate
def interleave(gate, up):
    n = gate.shape[0]
    return torch.stack([gate.reshape(n // 64, 64, -1), up.reshape(n // 64, 64, -1)], 1).reshape(2 * n, -1).contiguous()


@pytest.mark.parametrize("rows,im,block,parts", [(3, 20, 0, 1), (5, 128, 64, 1), (4, 36, 0, 3), (7, 192, 64, 2), (2, 9, 0, 2), (600, 64, 0, 1)])
@pytest.mark.parametrize("out_type", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("limit", [0.4, 7.0])
def test_clamped_gate_of_a_product(rows, im, block, parts, out_type, limit):
    g = torch.Generator().manual_seed(im)
    gate, up = 3.0 * torch.randn(rows, im, generator=g), 3.0 * torch.randn(rows, im, generator=g)
    gate[0, 0], up[0, 0], gate[0, 1], up[0, 1] = 50.0, -50.0, -50.0, 50.0
    gu = interleave(gate.T, up.T).T if block else torch.cat([gate, up], 1)
    src = gu.contiguous() if parts == 1 else torch.stack([0.5 * gu] + [0.5 * gu / (parts - 1)] * (parts - 1)).contiguous()
    out = torch.full((rows, im), NAN, device=DEV, dtype=out_type)
    ops().swiglu(dev(src), out, block, "glu_clamped", limit)
    assert rel_err(out, plain.cut_gate(gate.double(), up.double(), limit)) < (2e-6 if out_type == torch.float32 else 5e-3)


@pytest.mark.parametrize("T,im,K,splits", [(1, 64, 128, 1), (8, 320, 192, 2), (16, 128, 1536, 8), (13, 256, 520, 1)])
@pytest.mark.parametrize("limit", [0.3, 1.1])
def test_clamped_gate_inside_the_product_of_few_rows(T, im, K, splits, limit):
    g = torch.Generator().manual_seed(T + im)
    x = torch.randn(T, K, generator=g).to(torch.bfloat16)
    gate, up = ((torch.randn(im, K, generator=g) / math.sqrt(K)).to(torch.bfloat16) for _ in range(2))
    status = ops().new_status(DEV)
    out = torch.full((T, im), NAN, device=DEV, dtype=torch.bfloat16)
    ops().gemm_fused(dev(interleave(gate, up)), out, ops().FUSED_SWIGLU, x=dev(x), splits=splits, status=status, limit=limit)
    ops().raise_on_status(status)
    want = plain.cut_gate(x.double() @ gate.double().T, x.double() @ up.double().T, limit)
    assert rel_err(out, want) < 1e-2
    plain_out = torch.full((T, im), NAN, device=DEV, dtype=torch.bfloat16)           # without a limit: silu
    ops().gemm_fused(dev(interleave(gate, up)), plain_out, ops().FUSED_SWIGLU, x=dev(x), splits=splits, status=status)
    a, b = x.double() @ gate.double().T, x.double() @ up.double().T
    assert rel_err(plain_out, a / (1.0 + torch.exp(-a)) * b) < 1e-2


@pytest.mark.parametrize("T,im,K", [(256, 128, 64), (300, 320, 200), (999, 64, 136), (2048, 1024, 512)])
@pytest.mark.parametrize("limit", [0.3, 1.1])
def test_clamped_gate_inside_the_product_of_many_rows(T, im, K, limit):
    g = torch.Generator().manual_seed(T + im)
    x = torch.randn(T, K, generator=g).to(torch.bfloat16)
    gate, up = ((torch.randn(im, K, generator=g) / math.sqrt(K)).to(torch.bfloat16) for _ in range(2))
    status = ops().new_status(DEV)
    out = torch.full((T, im), NAN, device=DEV, dtype=torch.bfloat16)
    ops().gemm_pair(dev(x), dev(interleave(gate, up)), out, ops().PAIR_GLU_CLAMPED, None, status, limit=limit)
    ops().raise_on_status(status)
    assert rel_err(out, plain.cut_gate(x.double() @ gate.double().T, x.double() @ up.double().T, limit)) < 1e-2


# ---------------------------------------------------------------------------------------------- latent attention
@pytest.mark.parametrize("H,T,vd", [(3, 5, 7), (4, 40, 64), (1, 300, 16), (5, 3, 24)])
@pytest.mark.parametrize("dtype,gate_type", [(torch.float32, torch.float32), (torch.bfloat16, torch.float32), (torch.bfloat16, torch.bfloat16)])
def test_a_gate_for_every_feature_of_head_major_results(H, T, vd, dtype, gate_type):
    g = torch.Generator().manual_seed(H + T)
    src = torch.randn(H, T, vd, generator=g).to(dtype)
    gate = (2.0 * torch.randn(T, 16 + H * vd + (-H * vd) % 16, generator=g)).to(gate_type)
    out = torch.full((T, H * vd), NAN, device=DEV, dtype=dtype)
    ops().gate_heads(dev(src), dev(gate), 16, out, per_feature=True)
    want = src.double().transpose(0, 1).reshape(T, H * vd) * torch.sigmoid(gate[:, 16:16 + H * vd].double())
    assert rel_err(out, want) < (2e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("q_rank,rank,rot,rot_dims", [(72, 104, 0, 0), (768, 384, 0, 0), (0, 512, 64, 64), (12, 20, 6, 4), (11, 17, 0, 0),
                                                      (2048, 512, 64, 32)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_both_latents_normed_and_the_cached_row_appended(q_rank, rank, rot, rot_dims, dtype):
    T, page = 13, 8
    g = torch.Generator().manual_seed(rank)
    src = 2.0 * torch.randn(T, 16 + q_rank + rank + rot + 8, generator=g)
    src[:, :16] = NAN
    wq, w = (1 + 0.2 * torch.randn(max(q_rank, 1), generator=g)).to(dtype), (1 + 0.2 * torch.randn(rank, generator=g)).to(dtype)
    pos, req = [20 + t for t in range(9)] + [3, 4, 5, 6], [0] * 9 + [1] * 4
    cs = torch.randn(T, max(rot_dims // 2, 1), 2, generator=g)
    table = i32([[7, 3, 1, 9], [0, 2, 4, 5]])
    pool = torch.full((10, page, rank + rot), NAN, dtype=dtype, device=DEV)
    qo = torch.full((T, max(q_rank, 1)), NAN, dtype=dtype, device=DEV)
    status = ops().new_status(DEV)
    ops().latent_append(dev(src), 16 + q_rank, rank, rot, rot_dims, dev(w), 1e-4, dev(cs) if rot_dims else None, i32(pos), i32(req), table,
                        pool, status, q_norm=(16, dev(wq), qo) if q_rank else None)
    ops().raise_on_status(status)
    tol = 2e-6 if dtype == torch.float32 else 5e-3
    if q_rank:
        assert rel_err(qo, plain.rms_norm(src[:, 16:16 + q_rank].double(), wq.double(), 1e-4)) < tol
    c = plain.rms_norm(src[:, 16 + q_rank:16 + q_rank + rank].double(), w.double(), 1e-4)
    kr = src[:, 16 + q_rank + rank:16 + q_rank + rank + rot].double()
    turned = kr.clone()
    for i in range(rot_dims // 2):
        u, x, cc, s = kr[:, 2 * i], kr[:, 2 * i + 1], cs[:, i, 0].double(), cs[:, i, 1].double()
        turned[:, 2 * i], turned[:, 2 * i + 1] = u * cc - x * s, x * cc + u * s
    rows = torch.stack([pool[int(table[r, p // page]), p % page] for r, p in zip(req, pos)])
    assert rel_err(rows, torch.cat([c, turned], 1)) < tol
    assert int(torch.isnan(pool.float()).all(-1).sum()) == 10 * page - T


LATENT = [  # heads, latent, rotated part, page, window, positions, queries: rows of 16, 32 and 64 in a CTA, one and two tiles of keys in it
    (5, 512, 0, 16, 301, 700, 1), (12, 384, 0, 64, 0, 900, 1), (3, 384, 64, 64, 130, 500, 1), (16, 448, 0, 32, 0, 700, 1),
    (2, 512, 64, 64, 0, 600, 7), (5, 160, 0, 16, 0, 400, 60), (40, 256, 0, 64, 72, 300, 3), (6, 128, 32, 8, 0, 1100, 1), (1, 32, 0, 64, 3, 70, 70),
    (5, 448, 0, 16, 301, 700, 180),        # (every row a CTA of its own: more CTAs than leave room for two tiles in each)
]


@pytest.mark.parametrize("case", LATENT, ids=["-".join(map(str, c)) for c in LATENT])
@pytest.mark.parametrize("kernel", ["mma", "cuda_cores", "float"])
@pytest.mark.parametrize("sinks", [True, False])
def test_latent_attention_over_many_tiles(case, kernel, sinks):
    """The kernels that score against the cached rows themselves, over ranges of several tiles of keys, with keys that stand out
    in every tile so that a tile taken twice or left out shows; NaN in all that may not be read."""
    H, rank, rot, page, window, S, T = case
    o = ops()
    dtype = torch.float32 if kernel == "float" else torch.bfloat16
    g = torch.Generator().manual_seed(S + H)
    width, first = rank + rot, S - T
    rows = torch.randn(S, width, generator=g).to(dtype)
    q_lat = torch.randn(H, T, rank, generator=g)
    q_raw = torch.randn(T, H * (8 + rot), generator=g).to(dtype)
    for p in range(7, S, 50):                                   # every head looks for some of these
        h = p % H
        qq = torch.cat([q_lat[h, 0], q_raw.view(T, H, 8 + rot)[0, h, 8:].float()])
        rows[p] = (1.5 * qq * math.sqrt(width) / qq.norm()).to(dtype)
    q_lat = 0.3 * q_lat + q_lat[:, :1]
    sink = 2.0 * torch.randn(H, generator=g) + 2.0 if sinks else None
    scale = 2.0 / math.sqrt(width)
    lo = max(0, first - window + 1) if window else 0
    n_pages = -(-S // page)
    order = torch.randperm(n_pages + 2, generator=g).tolist()
    pool = torch.full((n_pages + 2, page, width), NAN).to(dtype)
    table = torch.full((1, n_pages + 2), -1, dtype=torch.int32)
    for i in range(n_pages):
        if (i + 1) * page > lo:
            table[0, i] = order[i]
            pool[order[i], :min(page, S - i * page)] = rows[i * page:i * page + min(page, S - i * page)]
    r, tile = o.latent_attention_plan(rank, rot)
    stages = 0
    if kernel == "mma":
        r, stages = o.latent_attention_mma_plan(rank, rot)
    hc = min(H, r)
    bq = 1 if T == 1 or T == 180 else max(1, r // hc)
    qblk = i32([[0, t, min(bq, T - t)] for t in range(0, T, bq)])
    out = torch.full((H, T, rank), NAN, dtype=dtype, device=DEV)
    status = o.new_status(DEV)
    o.latent_attention(dev(q_lat), dev(q_raw), 8, rot, 0, None, dev(pool), dev(table), i32(list(range(first, S))), qblk, qblk.shape[0],
                       S - 1, bq, hc, tile, 256, scale, out, status, mma_stages=stages, window=window,
                       sink_weight=None if sink is None else dev(sink))
    o.raise_on_status(status)
    full = torch.cat([q_lat.double().transpose(0, 1), q_raw.double().view(T, H, 8 + rot)[:, :, 8:]], -1)
    k = rows.double()
    want = torch.zeros(H, T, rank, dtype=torch.float64)
    for t in range(T):
        keys = plain.visible(first + t, window or None)
        p = plain.plain_softmax_weights((k[keys][:, None, :] * full[t]).sum(-1) * scale, None if sink is None else sink.double())
        want[:, t] = (p[:, :, None] * k[keys][:, None, :rank]).sum(0)
    assert rel_err(out, want) < (2e-5 if kernel == "float" else 2e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,rank", [(64, 64), (24, 40)])
def test_a_key_inside_and_outside_the_window_and_the_sink(tmp_path, dtype, dim, rank):
    """One latent layer whose every query looks for one token: it is found at the window's last place and not one further on, in a
    prompt (of 150 rows: in bfloat16 with heads of 64 through keys made per head) and in decoding; and a head whose sink lies far
    above every score gives nothing."""
    size = 37
    cfg = config(40, 64, 1e-6, [layer(lat(2, dim, dim, 32, rank, 1.0, window=size))])
    t = lively_tensors(cfg, 5, torch.float32)
    t["l0.mix.sink"] = torch.tensor([0.0, 60.0])
    # queries: a constant direction of the query latent; keys: the latent's first feature, which one token alone carries
    for name in ("l0.mix.dq", "l0.mix.uq", "l0.mix.dkv", "l0.mix.uk"):
        t[name].zero_()
    t["embed"][:, 0], t["embed"][:, 1] = 1.0, 0.0
    t["embed"][7, 1] = 1.5
    t["l0.mix.dq"][0, 0] = 1.0
    t["l0.mix.uq"][0, 0] = t["l0.mix.uq"][dim, 0] = 2.0
    t["l0.mix.dkv"][0, 1] = 1.0
    t["l0.mix.dkv"][1:9, 2:10] = torch.eye(8) * 0.5
    t["l0.mix.uk"][0, 0] = t["l0.mix.uk"][dim, 0] = 2.0
    stored = torch.float32 if dtype == "float32" else torch.bfloat16
    folder = write_model(str(tmp_path / "m"), cfg, {k: v.to(stored) for k, v in t.items()})
    from beglin_b200 import Engine
    ids = [11, 12, 13, 14, 15] * 30
    p = 60
    ids[p] = 7
    want = plain_logits(folder, ids)
    other = list(ids)
    other[p] = 16
    reach = (want - plain_logits(folder, other)).abs().amax(1) / want.abs().max()
    assert float(reach[p + size - 1]) > 0.1 and float(reach[p + size]) == 0.0
    tol = 5e-5 if dtype == "float32" else 3e-2
    eng = Engine.from_folder(folder, dtype=dtype, max_tokens=192, page_size=16, max_requests=2)
    whole = eng.step([("w", ids, list(range(len(ids))))], end=["w"])
    assert rel_err(whole, want) < tol
    head = p + size - 4
    eng.step([("d", ids[:head], [])])
    for i in range(head, head + 8):
        row = eng.step([("d", [ids[i]], [0])])
        assert rel_err(row[0], want[i]) < tol * float(want.abs().max() / want[i].abs().max()), i
