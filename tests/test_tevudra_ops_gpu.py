"""Each mechanism of the Tevudra design alone, against the plain functions of ``oracle/tevudra.py``."""
import math

import numpy as np
import pytest
import torch

from conftest import load
from oracle import tevudra as ot

pytestmark = pytest.mark.gpu

BF, F32 = torch.bfloat16, torch.float32


def gen(seed):
    return torch.Generator().manual_seed(seed)


def close(got, want, dtype, bf=2e-2, f32=2e-5):
    got, want = got.double().cpu(), want.double().cpu()
    err = (got - want).abs().max() / want.abs().max().clamp(min=1e-9)
    assert float(err) <= (bf if dtype == BF else f32), float(err)


# ---------------------------------------------------------------- feed-forward activations in the projection
@pytest.mark.parametrize("T", [1, 5, 33, 300])
@pytest.mark.parametrize("act", ["relu2", "gelu"])
def test_projection_activations(ops, cuda, T, act):
    g = gen(T)
    x, W = torch.randn(T, 72, generator=g).bfloat16(), torch.randn(200, 72, generator=g).bfloat16() / 8
    flag, fn = (ops.ACT_RELU2, ot.relu2) if act == "relu2" else (ops.ACT_GELU, ot.gelu_erf)
    want = fn(x.double() @ W.double().T)
    close(ops.linear(x.to(cuda), ops.PackedWeight(W.to(cuda)), flags=flag), want, BF)
    close(ops.linear(x.to(cuda), W.to(cuda), flags=flag | ops.FORCE_SIMT), want, BF)
    close(ops.linear_f32(x.float().to(cuda), W.float().to(cuda), flag), want, F32)


# ---------------------------------------------------------------- dynamic tanh norm
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,H", [(1, 8), (3, 88), (65, 2056), (7, 4096)])
def test_residual_dyt(ops, cuda, dtype, T, H):
    g = gen(T + H)
    r, d = torch.randn(T, H, generator=g), torch.randn(T, H, generator=g).to(dtype)
    w, b = torch.randn(H, generator=g).bfloat16(), torch.randn(H, generator=g).bfloat16()
    alpha = torch.tensor([0.7]).bfloat16()
    norm = lambda x: ot.dyt(x, alpha.double(), w.double(), b.double())
    dev = lambda t: t.to(cuda)
    res, out = dev(r.clone()), torch.empty(T, H, dtype=dtype, device=cuda)
    ops.residual_dyt(None, res, dev(w), dev(b), dev(alpha), out)
    assert torch.equal(res.cpu(), r)
    close(out, norm(r.double()), dtype, bf=6e-3)
    ops.residual_dyt(dev(d), res, dev(w), dev(b), dev(alpha), out)
    total = r.double() + d.double()
    close(res, total, F32)
    close(out, norm(total), dtype, bf=6e-3)
    rows = torch.tensor(sorted({0, T // 2, T - 1}), dtype=torch.int32)
    out2 = torch.empty(len(rows), H, dtype=dtype, device=cuda)
    ops.residual_dyt(dev(d), res, dev(w), dev(b), dev(alpha), out2, rows=dev(rows))
    close(out2, norm(total[rows.long()] + d[rows.long()].double()), dtype, bf=6e-3)


# ---------------------------------------------------------------- routing
@pytest.mark.parametrize("T,E,top,tile", [(1, 1, 1, 16), (1, 11, 2, 16), (5, 7, 7, 32), (32, 70, 6, 16), (2, 300, 8, 64),
                                          (900, 5, 2, 256), (700, 64, 6, 128), (3000, 9, 1, 64), (1024, 2, 2, 16)])
def test_moe_plan(ops, cuda, T, E, top, tile):
    g = gen(E * T)
    z, b = torch.randn(T, E + 3, generator=g), torch.randn(E, generator=g)
    z[0, :E] = 0.0
    b[: E // 2] = 0.5  # equal logits in token 0: the lower index first
    plan = ops.MoePlan(T, E, top, cuda)
    ops.moe_plan(z.to(cuda), b.to(cuda), plan, T, tile)
    _check_plan(plan, z[:, :E] + b, T, E, top, tile)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,E,top,width", [(1, 1, 1, 8), (1, 11, 2, 40), (5, 7, 7, 320), (32, 70, 6, 264), (64, 300, 8, 1000), (64, 5, 3, 72)])
def test_moe_route_plan_in_one_launch(ops, cuda, dtype, T, E, top, width):
    g = gen(E + T)
    # small integers: the logits are exact in fp32 whatever the order of the sum
    h, W = (torch.randint(-3, 4, s, generator=g).to(dtype) for s in ((T, width), (E, width)))
    b = torch.randn(E, generator=g)
    plan = ops.MoePlan(T, E, top, cuda)
    for _ in range(2):  # (the ticket resets itself)
        ops.moe_route_plan(h.to(cuda), W.to(cuda), b.to(cuda), plan, 16)
        _check_plan(plan, h.float() @ W.float().T + b, T, E, top, 16)


def _check_plan(plan, total, T, E, top, tile):
    order = torch.sort(total, dim=-1, descending=True, stable=True)
    idx, wt = plan.expert[:T * top].cpu().view(T, top), plan.weight[:T * top].cpu().view(T, top)
    assert torch.equal(idx.long(), order.indices[:, :top])
    torch.testing.assert_close(wt, torch.softmax(order.values[:, :top].double(), -1).float(), atol=2e-6, rtol=2e-6)
    flat = idx.flatten().numpy()
    by_expert = np.argsort(flat, kind="stable")  # pairs of an expert stay in token order
    pos, rows = plan.pos[:T * top].cpu().numpy(), plan.rows[:T * top].cpu().numpy()
    assert np.array_equal(pos[by_expert], np.arange(T * top)) and np.array_equal(rows, by_expert // top)
    tiles = plan.tiles.cpu().numpy()
    want, first = [], 0
    for e in range(E):
        n = int((flat == e).sum())
        want += [(e, first + r, min(tile, n - r), 0) for r in range(0, n, tile)]
        first += n
    assert tiles[0] == len(want) <= plan.max_tiles
    assert np.array_equal(tiles[4:4 + 4 * len(want)].reshape(-1, 4), np.asarray(want))


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,E,top,width,ff,tile", [(1, 3, 2, 40, 24, 16), (9, 12, 3, 320, 136, 16), (40, 6, 2, 136, 72, 32),
                                                   (70, 3, 2, 200, 88, 64), (300, 4, 2, 192, 264, 128), (1100, 3, 2, 136, 144, 256)])
def test_grouped_experts_and_weighted_sum(ops, cuda, dtype, T, E, top, width, ff, tile):
    """Gathered up projection with gelu, down projection in expert order, weighted sum into the residual."""
    g = gen(T)
    r = lambda *s, k=1.0: (torch.randn(*s, generator=g) * k).bfloat16()
    h, rw, rb = r(T, width), r(E, width, k=width ** -0.5), r(E)
    ex = [(r(ff, width, k=width ** -0.5), r(width, ff, k=ff ** -0.5)) for _ in range(E)]
    d64 = lambda t: t.double()
    z = d64(h) @ d64(rw).T
    want = ot.moe(d64(h), d64(rw), d64(rb), top, [(d64(a), d64(b)) for a, b in ex])
    stack = lambda i: ops.GroupedWeight(torch.stack([e[i] for e in ex]).to(dtype).to(cuda))
    up, down = stack(0), stack(1)
    plan = ops.MoePlan(T, E, top, cuda)
    if dtype == F32:
        tile = ops.F32_TILE_ROWS
    ops.moe_plan(z.float().to(cuda), rb.float().to(cuda), plan, T, tile)
    work = ops.new_workspace(ops._lib.lib().mlora_grouped_linear_workspace(tile), cuda)
    x = h.to(dtype).to(cuda)
    a = torch.full((T * top, ff), float("nan"), dtype=dtype, device=cuda)
    y = torch.full((T * top, width), float("nan"), dtype=dtype, device=cuda)
    for _ in range(2):  # (the scratch's counters reset themselves)
        ops.grouped_linear(x, up, a, plan=plan, gather=True, flags=ops.ACT_GELU, work=work)
        ops.grouped_linear(a, down, y, plan=plan, work=work)
    assert ops.status_word(work) == 0
    res, out = torch.zeros(T, width, device=cuda), torch.empty(T, width, dtype=dtype, device=cuda)
    one = torch.ones(width, dtype=BF, device=cuda)
    ops.residual_dyt(None, res, one, one, one[:1], out, expert_rows=y, plan=plan)
    close(res, want, dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,H,k,n,tile", [(1, 3, 64, 128, 16), (20, 5, 128, 384, 32), (33, 2, 512, 64, 64), (260, 3, 64, 136, 128)])
def test_grouped_heads_with_gates(ops, cuda, dtype, T, H, k, n, tile):
    """Every group the same rows, another column slice of x and y, outputs times a sigmoid gate per row and group."""
    g = gen(T + H)
    x, W, gate = (torch.randn(*s, generator=g).bfloat16() for s in ((T, H * k + 8), (H, n, k), (T, H + 4)))
    W = W / 8
    want = torch.einsum("thk,hnk->thn", x[:, :H * k].double().view(T, H, k), W.double())
    want = (want * torch.sigmoid(gate[:, :H].double())[:, :, None]).flatten(1)
    y = torch.full((T, H * n), float("nan"), dtype=dtype, device=cuda)
    work = ops.new_workspace(ops._lib.lib().mlora_grouped_linear_workspace(tile), cuda)
    ops.grouped_linear(x.to(dtype).to(cuda), ops.GroupedWeight(W.to(dtype).to(cuda)), y, T=T, x_cols=k, y_cols=n, tile_rows=tile,
                       gate=gate.to(dtype).to(cuda), work=work)
    close(y, want, dtype)


# ---------------------------------------------------------------- latents in pages
def tile(pages):
    """Row-major pages to the stored order, element by element from its definition."""
    n, ps, pitch = pages.shape
    row, k = torch.meshgrid(torch.arange(ps), torch.arange(pitch), indexing="ij")
    chunk = ((k % 64) // 8) ^ (row % 8)
    off = (row // 8) * 8 * pitch + (k // 64) * 512 + (row % 8) * 64 + chunk * 8 + k % 8
    out = torch.empty(n, ps * pitch, dtype=pages.dtype)
    out[:, off.flatten()] = pages.flatten(1)
    return out.view(n, ps, pitch)


class Pages:
    """Scrambled page table over sequences of the given lengths; every place no sequence uses holds NaN."""

    def __init__(self, lens, R, ps, dtype, dev, seed=0):
        g = gen(seed)
        self.lens, self.R, self.ps, self.pitch = lens, R, ps, -(-R // 64) * 64
        need = [-(-n // ps) for n in lens]
        self.max_pages = max(need) + 2
        ids = torch.randperm(sum(need) + 3, generator=g).tolist()
        self.pages = torch.full((sum(need) + 3, ps, self.pitch), float("nan"), dtype=dtype)
        self.bt = torch.full((len(lens), self.max_pages), ids[-1], dtype=torch.int32)
        self.c = [torch.randn(n, R, generator=g).to(dtype) for n in lens]
        it = iter(ids)
        for s, n in enumerate(lens):
            for p in range(need[s]):
                self.bt[s, p] = next(it)
        self.dev = dev

    def fill(self):
        for s, c in enumerate(self.c):
            for j in range(len(c)):
                row = self.pages[self.bt[s, j // self.ps], j % self.ps]
                row[: self.R], row[self.R:] = c[j], 0
        return tile(self.pages).to(self.dev), self.bt.to(self.dev)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("R,col", [(3, 5), (30, 5), (128, 8), (264, 16), (512, 0), (96, 8), (264, 3), (520, 8)])
def test_latent_append_and_gather(ops, cuda, dtype, R, col):
    lens = [1, 16, 17, 40]
    pg = Pages(lens, R, 16, dtype, cuda)
    pages, bt = pg.pages.clone().to(cuda), pg.bt.to(cuda)
    slot = torch.tensor([s for s, n in enumerate(lens) for _ in range(n)] + [0], dtype=torch.int32)
    pos = torch.tensor([j for n in lens for j in range(n)] + [-1], dtype=torch.int32)  # the last row is padding
    perm = torch.randperm(len(slot), generator=gen(1))
    x = torch.randn(len(slot), -(-(R + col) // 8) * 8, generator=gen(2)).to(dtype)
    w = torch.randn(R, generator=gen(3)).bfloat16()
    ops.latent_append(x[perm].to(cuda)[:, col:], R, w.to(cuda), 0.1, pages, bt, slot[perm].to(cuda), pos[perm].to(cuda))
    want = ot.rms(x[:, col:col + R].double(), w.double(), 0.1)
    got = load("kv_cache").PagedLatentCache.untile(pages.cpu())
    assert torch.equal(torch.nan_to_num(tile(got), nan=7.0), torch.nan_to_num(pages.cpu(), nan=7.0))
    used = torch.zeros(got.shape[:2], dtype=torch.bool)
    for i in range(len(slot) - 1):
        p, o = int(pg.bt[slot[i], pos[i] // 16]), int(pos[i]) % 16
        used[p, o] = True
        close(got[p, o, :R], want[i], dtype, bf=5e-3, f32=1e-6)
        assert (got[p, o, R:] == 0).all()
    assert torch.isnan(got[~used].float()).all()  # nothing else was written
    if dtype == BF:
        segs = torch.tensor([(2, 0, 17, 0), (3, 32, 40, 0), (0, 80, 1, 0)], dtype=torch.int32)
        dense = torch.zeros(96, pg.pitch, dtype=dtype, device=cuda)
        ops.latent_gather(pages, bt, segs.to(cuda), 3, 48, dense)
        for s, base, n, _ in segs.tolist():
            for j in range(n):
                assert torch.equal(dense[base + j].cpu(), got[pg.bt[s, j // 16], j % 16])


def _latent_reference(pg, qa, slot, pos, H, scale):
    out = []
    for i in range(len(slot)):
        if pos[i] < 0:
            out.append(torch.zeros(H, pg.R, dtype=torch.float64))
            continue
        c = pg.c[slot[i]][: pos[i] + 1].double()
        p = torch.softmax(qa[i, :, : pg.R].double() @ c.T * scale, -1)
        out.append(p @ c)
    return torch.stack(out)


def _run_latent(ops, cuda, pg, H, rows, scale, dtype, splits, simt, spike):
    slot, pos = [r[0] for r in rows], [r[1] for r in rows]
    rq = -(-pg.R // 128) * 128
    qa = torch.zeros(len(rows), H, rq)
    qa[:, :, : pg.R] = torch.randn(len(rows), H, pg.R, generator=gen(7)) / math.sqrt(pg.R)
    for i, (s, p, *key) in enumerate(rows):
        if key:  # this key's score stands out in every head
            qa[i, :, : pg.R] = pg.c[s][key[0]].float() * spike / float(pg.c[s][key[0]].float().pow(2).sum())
    qa = qa.to(dtype)
    want = _latent_reference(pg, qa, slot, pos, H, scale)
    pages, bt = pg.fill()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=cuda)
    out = torch.full((len(rows), H * rq), float("nan"), dtype=dtype, device=cuda)
    nb = ops.latent_attention_workspace(len(rows), H, rq, splits)
    status = torch.zeros(1, dtype=torch.int32, device=cuda)
    ops.latent_attention(qa.flatten(1).to(cuda), pg.R, H, pages, bt, i32(slot), i32(pos), scale, out, n_splits=splits,
                         work=ops.new_workspace(nb, cuda), status=status, simt=simt)
    assert int(status) == 0
    got = out.cpu().view(len(rows), H, rq)
    assert (got[:, :, pg.R:] == 0).all()
    close(got[:, :, : pg.R], want, dtype, bf=1.5e-2)
    # row by row as well: a short context must not hide behind a long one
    for i in range(len(rows)):
        if pos[i] >= 0:
            close(got[i, :, : pg.R], want[i], dtype, bf=2.5e-2, f32=5e-5)


EDGES = [1, 2, 15, 16, 17, 127, 128, 129, 255, 256, 257, 400]


@pytest.mark.parametrize("ps", [16, 32])
@pytest.mark.parametrize("splits", [1, 2, 3, 7])
def test_latent_attention_at_page_block_and_split_borders(ops, cuda, ps, splits):
    pg = Pages(EDGES, 72, ps, BF, cuda, seed=ps)
    _run_latent(ops, cuda, pg, 5, [(s, n - 1) for s, n in enumerate(EDGES)] + [(0, -1)], 1.3, BF, splits, False, 0)


@pytest.mark.parametrize("R,H", [(8, 1), (64, 16), (96, 17), (128, 32), (200, 33), (256, 6), (320, 70), (512, 32), (500, 4)])
def test_latent_attention_ranks_and_head_groups(ops, cuda, R, H):
    lens = [300, 5, 140]
    pg = Pages(lens, R, 16, BF, cuda, seed=R)
    rows = [(0, 299), (1, 4), (2, 139), (0, 128), (0, 127)]
    for splits in (1, 2):
        _run_latent(ops, cuda, pg, H, rows, 2.0, BF, splits, False, 0)


@pytest.mark.parametrize("dtype,R,H", [(BF, 520, 3), (BF, 40, 20), (F32, 44, 3), (F32, 640, 2), (F32, 2048, 1)])
def test_latent_attention_on_cuda_cores(ops, cuda, dtype, R, H):
    lens = [1, 16, 63, 64, 65, 130]
    pg = Pages(lens, R, 16, dtype, cuda, seed=R)
    rows = [(s, n - 1) for s, n in enumerate(lens)] + [(5, 100), (3, -1)]
    _run_latent(ops, cuda, pg, H, rows, 0.9, dtype, 1, True, 0)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_latent_attention_one_key_stands_out(ops, cuda, dtype):
    """One key decides, wherever it lies: the first, the last visible, page and block borders; and the running maximum
    jumps by tens at that key, in every block order."""
    n = 390
    pg = Pages([n], 64, 16, dtype, cuda)
    keys = [0, 1, 15, 16, 127, 128, 129, 255, 256, 383, 384, 388, 389]
    rows = [(0, n - 1, k) for k in keys] + [(0, k, k) for k in keys] + [(0, k, 0) for k in keys]
    for splits in (1, 3):
        _run_latent(ops, cuda, pg, 4, rows, 1.0, dtype, splits, dtype == F32, 40.0)
    # the key just after the last visible one must not matter
    pg.c[0][200] = 30.0
    _run_latent(ops, cuda, pg, 4, [(0, 199), (0, 150)], 1.0, dtype, 1, dtype == F32, 0)


def test_latent_attention_negative_scale(ops, cuda):
    pg = Pages([150], 72, 16, BF, cuda)
    _run_latent(ops, cuda, pg, 3, [(0, 149), (0, 128)], -1.5, BF, 1, False, 0)


# ---------------------------------------------------------------- prompt attention over expanded keys and values
@pytest.mark.parametrize("dk,dv", [(64, 64), (64, 128), (128, 64), (128, 128)])
def test_prefill_attention_dense(ops, cuda, dk, dv):
    """Portions with and without a history, lengths at tile borders; keys of the neighbouring sequence lie right behind."""
    H, scale = 3, 1.7 / math.sqrt(dk)
    seqs = [(0, 1), (0, 130), (100, 28), (127, 2), (128, 128), (300, 5)]  # (history, new rows)
    g = gen(dk + dv)
    T = sum(n for _, n in seqs)
    q = torch.randn(T, H * dk + 16, generator=g).bfloat16()
    gate = torch.randn(T, H, generator=g).bfloat16()
    ctx = [-(-(p + n) // 16) * 16 for p, n in seqs]
    kv = torch.randn(sum(ctx), H * (dk + dv), generator=g).bfloat16()
    tiles, want, base, r0 = [], [], 0, 0
    for (p, n), c in zip(seqs, ctx):
        kv[base + p + n: base + c] = float("nan")  # the tail of a sequence's last page
        tiles += [(base, r0 + o, min(128, n - o), p + o) for o in range(0, n, 128)]
        k = kv[base: base + p + n, : H * dk].double().view(-1, H, dk)
        v = kv[base: base + p + n, H * dk:].double().view(-1, H, dv)
        s = torch.einsum("ihd,jhd->hij", q[r0:r0 + n, : H * dk].double().view(n, H, dk), k) * scale
        i, j = torch.arange(n)[:, None] + p, torch.arange(p + n)[None]
        w = torch.softmax(s.masked_fill(j > i, float("-inf")), -1)
        want.append((torch.einsum("hij,jhd->ihd", w, v) * torch.sigmoid(gate[r0:r0 + n].double())[:, :, None]).flatten(1))
        base, r0 = base + c, r0 + n
    out = torch.full((T, H * dv), float("nan"), dtype=BF, device=cuda)
    status = torch.zeros(1, dtype=torch.int32, device=cuda)
    ops.prefill_attention_dense(q.to(cuda), kv.to(cuda), H * dk, torch.tensor(tiles, dtype=torch.int32, device=cuda), len(tiles), H,
                                dk, dv, scale, out, gate=gate.to(cuda), status=status)
    assert int(status) == 0
    close(out, torch.cat(want), BF, bf=1.5e-2)
