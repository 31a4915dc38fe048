"""The grouped products over experts on tcgen05 against the products in 64-bit and against the mma.sync kernel: every kind,
tiles of few and of many rows, experts without a token, sizes that leave rests."""
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


SHAPES = [(1, 4, 2, 64, 32), (3, 12, 3, 320, 64), (9, 5, 1, 48, 24), (64, 16, 4, 256, 128), (150, 6, 2, 72, 200), (300, 3, 3, 1024, 512),
          (700, 16, 4, 128, 96), (40, 40, 7, 136, 18), (1500, 8, 2, 512, 136), (260, 1, 1, 8, 264)]


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
        old = torch.empty_like(out)
        K.moe_grouped(*args, old, **kw)
        assert float((out.double() - old.double()).abs().max()) <= 6e-3 * big
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
