"""The grouped products over experts on tcgen05 against the products in 64-bit: every kind, tiles of few and of many rows, experts without a token, sizes that leave rests."""
import pytest
import torch

pytestmark = pytest.mark.gpu


def _case(T, E, top, W, F, seed, skew=False):
    g = torch.Generator().manual_seed(seed)
    x = torch.randn(T, W, generator=g).to(torch.bfloat16)
    score = torch.rand(T, E, generator=g)
    if skew:                                       # one expert gets nearly every token, some get none
        score[:, 0] += 1.0
        score[:, E // 2:] -= 1.0
    ids = score.topk(top, dim=1).indices.to(torch.int32)
    gate, up = ((torch.randn(E, F, W, generator=g) / W ** 0.5 * 1.5).to(torch.bfloat16) for _ in range(2))
    down = (torch.randn(E, W, F, generator=g) / F ** 0.5).to(torch.bfloat16)
    return x, ids, gate, up, down, torch.rand(T, top, generator=g) + 0.5


def _expert(kind, act, limit, x, gate, up, wt):
    g, u = x @ gate.T * wt, x @ up.T * wt
    if kind == "up":
        return torch.clamp(u, min=0.0) ** 2
    if act == 1:
        return g * torch.sigmoid(g) * u
    g, u = torch.clamp(g, max=limit), torch.clamp(u, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


SHAPES = [(1, 4, 2, 64, 32), (3, 10, 3, 336, 80), (9, 5, 1, 48, 24), (64, 16, 4, 256, 128), (150, 6, 2, 72, 200), (300, 3, 3, 1024, 512),
          (700, 16, 4, 128, 96), (40, 40, 7, 136, 24), (1500, 8, 2, 512, 136), (260, 1, 1, 8, 264)]


@pytest.mark.parametrize("wide", [False, True])
@pytest.mark.parametrize("skew", [False, True])
@pytest.mark.parametrize("shape", SHAPES)
def test_the_tcgen05_grouped_products(shape, skew, wide, monkeypatch):
    from firefly_b200.ops import kernels as K
    T, E, top, W, F = shape
    if skew and top > (E + 1) // 2:
        pytest.skip("not enough experts for the skewed choice")
    monkeypatch.setattr(K, "MOE_WIDE_BLOCKS_PER_SM", 0 if wide else 1 << 20)
    x, ids, gate, up, down, wts = _case(T, E, top, W, F, T + E, skew)
    dev = [t.cuda() for t in (x, ids, gate, up, down, wts)]
    xd, idd, gd, ud, dd, wd = dev
    n = T * top
    tiles = K.moe_max_tiles(n, E, True)
    i32 = dict(dtype=torch.int32, device="cuda")
    seg, row_of, src, te, tr, nt = (torch.empty(k, **i32) for k in (E + 1, n, n, tiles, tiles, 1))
    row_w, status = torch.empty(n, device="cuda"), torch.zeros(1, **i32)
    torch.cuda.synchronize()
    K.moe_plan(idd, E, seg, row_of, src, te, tr, nt, True, wd, row_w)
    plan = (seg, te, tr, nt, tiles)
    order = torch.empty(n, dtype=torch.long)
    order[row_of.cpu().long()] = torch.arange(n)             # which (token, choice) each row is
    tok, ex, wt = order // top, ids.view(-1)[order].long(), wts.view(-1)[order].double()
    for kind, act, weighted in (("gate_up", 0, False), ("gate_up", 1, True), ("up", 0, True), ("up", 0, False)):
        out = torch.full((n, F), float("nan"), dtype=torch.bfloat16, device="cuda")
        args = (xd, src, gd if kind == "gate_up" else ud, ud if kind == "gate_up" else None, plan)
        kw = dict(limit=0.8, tensor_cores=True, act=act, kind=K.MOE_UP if kind == "up" else None, row_w=row_w if weighted else None)
        K.moe_grouped(*args, out, status=status, **kw)
        want = torch.empty(n, F, dtype=torch.float64)
        for e in range(E):
            m = ex == e
            want[m] = _expert(kind, act, 0.8, x[tok[m]].double(), gate[e].double(), up[e].double(), (wt[m] if weighted else torch.ones(int(m.sum()))).double()[:, None])
        big = float(want.abs().max())
        assert float((out.cpu().double() - want).abs().max()) <= 6e-3 * big, (kind, act, weighted)
        again = torch.empty_like(out)
        K.moe_grouped(*args, again, status=status, **kw)
        assert torch.equal(out, again)
    act_rows = (torch.randn(n, F, generator=torch.Generator().manual_seed(1))).to(torch.bfloat16)
    res = torch.full((n, W), float("nan"), device="cuda")
    K.moe_grouped(act_rows.cuda(), src, dd, None, plan, res, 0.0, True, status=status)
    want = torch.empty(n, W, dtype=torch.float64)
    for e in range(E):
        want[ex == e] = act_rows[ex == e].double() @ down[e].double().T
    assert float((res.cpu().double() - want).abs().max()) <= 2e-5 * float(want.abs().max())
    assert int(status[0]) == 0


def test_rows_do_not_depend_on_what_shares_their_tile(monkeypatch):
    """A token alone and among hundreds: the same bits from either width of tile."""
    from firefly_b200.ops import kernels as K
    T, E, top, W, F = 400, 6, 2, 256, 128
    x, ids, gate, up, down, wts = _case(T, E, top, W, F, 5)
    got = {}
    for wide in (False, True):
        monkeypatch.setattr(K, "MOE_WIDE_BLOCKS_PER_SM", 0 if wide else 1 << 20)
        for n_tok in (T, 3):
            xd, idd, gd, ud = x[:n_tok].cuda(), ids[:n_tok].contiguous().cuda(), gate.cuda(), up.cuda()
            n = n_tok * top
            tiles = K.moe_max_tiles(n, E, True)
            i32 = dict(dtype=torch.int32, device="cuda")
            seg, row_of, src, te, tr, nt = (torch.empty(k, **i32) for k in (E + 1, n, n, tiles, tiles, 1))
            out, status = torch.empty(n, F, dtype=torch.bfloat16, device="cuda"), torch.zeros(1, **i32)
            torch.cuda.synchronize()
            K.moe_plan(idd, E, seg, row_of, src, te, tr, nt, True)
            K.moe_grouped(xd, src, gd, ud, (seg, te, tr, nt, tiles), out, 0.8, True, status=status)
            got[wide, n_tok] = out[row_of.long()][: 3 * top].cpu()
            assert int(status[0]) == 0
    first = got[False, 3]
    assert all(torch.equal(first, v) for v in got.values())


@pytest.mark.parametrize("T,E,top", [(1, 3, 1), (5, 4, 4), (700, 11, 3), (1024, 16, 4), (1025, 16, 4), (3000, 300, 2), (16384, 16, 4), (2111, 5, 2)])
@pytest.mark.parametrize("tc", [True, False])
def test_the_plan_sorts_every_choice_by_expert(T, E, top, tc):
    """One block and a cluster of them: every (token, choice) has a row of its own in its expert's range, the rows' tokens and
    weights are its, and the row tiles cover the ranges."""
    from firefly_b200.ops import kernels as K
    g = torch.Generator().manual_seed(T + E)
    score = torch.rand(T, E, generator=g)
    score[:, E // 2] += 0.6                                  # uneven, and some experts without a row where there are few tokens
    ids = score.topk(top, dim=1).indices.to(torch.int32)
    wts = torch.rand(T, top, generator=g)
    n, tiles, rt = T * top, K.moe_max_tiles(T * top, E, tc), K.moe_row_tile(tc)
    i32 = dict(dtype=torch.int32, device="cuda")
    seg, row_of, src, te, tr, nt = (torch.full((k,), -7, **i32) for k in (E + 1, n, n, tiles, tiles, 1))
    row_w = torch.zeros(n, device="cuda")
    idd, wd = ids.cuda(), wts.cuda()
    torch.cuda.synchronize()
    K.moe_plan(idd, E, seg, row_of, src, te, tr, nt, tc, wd, row_w)
    seg, row_of, src, te, tr, row_w = (t.cpu() for t in (seg, row_of, src, te, tr, row_w))
    counts = torch.bincount(ids.view(-1).long(), minlength=E)
    assert torch.equal(seg.long(), torch.cat([torch.zeros(1, dtype=torch.long), counts.cumsum(0)]))
    assert torch.equal(row_of.long().sort().values, torch.arange(n))
    e = ids.view(-1).long()
    assert bool(((row_of >= seg[e]) & (row_of < seg[e + 1])).all())
    assert torch.equal(src[row_of.long()].long(), torch.arange(n) // top) and torch.equal(row_w[row_of.long()], wts.view(-1))
    want = [(k, int(seg[k]) + r) for k in range(E) for r in range(0, int(counts[k]), rt)]
    assert int(nt[0]) == len(want) <= tiles and list(zip(te.tolist(), tr.tolist()))[: len(want)] == want


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,F", [(1, 8), (3, 21), (64, 1024), (513, 40), (7, 36)])
def test_the_clamped_activation(dtype, T, F):
    from firefly_b200.ops import kernels as K
    gu = (torch.randn(T, 2 * F, generator=torch.Generator().manual_seed(F)) * 2).to(dtype)
    y = torch.empty(T, F, dtype=dtype, device="cuda")
    K.clamped_glu(gu.cuda(), y, 1.25)
    g, u = torch.clamp(gu[:, :F].double(), max=1.25), torch.clamp(gu[:, F:].double(), min=-1.25, max=1.25)
    want = g * torch.sigmoid(1.702 * g) * (u + 1.0)
    assert float((y.cpu().double() - want).abs().max()) <= (2e-6 if dtype == torch.float32 else 5e-3) * float(want.abs().max())
