"""Each mechanism of the Relidra design alone, against the plain functions of ``oracle/relidra.py``."""
import numpy as np
import pytest
import torch

from conftest import load
from oracle import relidra as orl

pytestmark = pytest.mark.gpu

BF, F32 = torch.bfloat16, torch.float32


def gen(seed):
    return torch.Generator().manual_seed(seed)


def close(got, want, dtype, bf=2e-2, f32=2e-5):
    got, want = got.double().cpu(), want.double().cpu()
    err = (got - want).abs().max() / want.abs().max().clamp(min=1e-9)
    assert float(err) <= (bf if dtype == BF else f32), float(err)


def i32(v, cuda):
    return torch.as_tensor(np.asarray(v, dtype=np.int32), device=cuda)


# ---------------------------------------------------------------- hyper-connections + layer norm
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,n,width", [(1, 1, 8), (3, 2, 84), (5, 3, 1000), (33, 4, 4096), (2, 7, 300), (2, 16, 2048), (3, 2, 11000)])
def test_streams_and_layer_norm(ops, cuda, dtype, T, n, width):
    g = gen(T + n)
    H = -(-width // 8) * 8
    pad = lambda t: torch.nn.functional.pad(t, (0, H - width))
    x = torch.randn(T, n, width, generator=g) + 3  # (a mean that matters)
    y = torch.randn(T, width, generator=g).to(dtype)
    w = torch.randn(width, generator=g).bfloat16()
    read, out_w, mix = torch.rand(n, generator=g), torch.randn(n, generator=g), torch.randn(n, n, generator=g)
    back = torch.cat([out_w, mix.flatten()]).to(cuda)
    D = lambda t: t.double()
    ln = lambda u: orl.layer_norm(u, D(w), 0.01)
    dev = lambda t: pad(t).contiguous().to(cuda)
    o = torch.full((T, H), float("nan"), dtype=dtype, device=cuda)
    args = (dev(w), 0.01, width, o)
    # a first sublayer: all streams are one row, nothing comes back
    same = dev(x[:, 0])
    ops.residual_streams_layernorm(None, same, read.to(cuda), *args)
    close(o[:, :width], ln(D(read).sum() * D(x[:, 0])), dtype, bf=6e-3)
    assert not o[:, width:].any()
    # its result: the streams part ways
    streams = torch.full((T, n, H), float("nan"), device=cuda)
    ops.residual_streams_layernorm(dev(y), same, read.to(cuda), *args, dst=streams, back=back)
    want = orl.hyper_connect(D(x[:, :1]).expand(-1, n, -1).transpose(0, 1), D(read), D(mix), D(out_w), lambda u: D(y))
    close(streams[:, :, :width].transpose(0, 1), want, F32)
    close(o[:, :width], ln(torch.einsum("s,stw->tw", D(read), want)), dtype, bf=6e-3)
    # in place
    streams.copy_(dev(x))
    ops.residual_streams_layernorm(dev(y), streams, read.to(cuda), *args, dst=streams, back=back)
    want = orl.hyper_connect(D(x).transpose(0, 1), D(read), D(mix), D(out_w), lambda u: D(y))
    close(streams[:, :, :width].transpose(0, 1), want, F32)
    close(o[:, :width], ln(torch.einsum("s,stw->tw", D(read), want)), dtype, bf=6e-3)
    assert not streams[:, :, width:].any()
    # the end: the sum of the streams, some rows only, nothing kept
    streams.copy_(dev(x))
    rows = torch.tensor(sorted({T - 1, T // 2, 0}, reverse=True), dtype=torch.int32)
    o2 = torch.empty(len(rows), H, dtype=dtype, device=cuda)
    ops.residual_streams_layernorm(dev(y), streams, torch.ones(n, device=cuda), dev(w), 0.01, width, o2, back=back, rows=rows.to(cuda))
    close(o2[:, :width], ln(want.sum(0)[rows.long()]), dtype, bf=6e-3)
    assert torch.equal(streams.cpu(), pad(x))


# ---------------------------------------------------------------- rotation, norm, append
def _table(g, n_seq, pages_each, cuda):
    ids = torch.randperm(n_seq * pages_each + 3, generator=g)[:n_seq * pages_each].view(n_seq, pages_each)
    return ids.to(torch.int32).to(cuda), n_seq * pages_each + 3


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("Hq,Hkv,dim,rot,pad,page,factor", [(4, 2, 36, 20, 64, 16, 2.5), (5, 1, 72, 72, 128, 32, 1.0), (3, 3, 9, 0, 16, 16, 1.0),
                                                            (1, 1, 144, 100, 144, 16, 4.0), (8, 2, 128, 128, 128, 16, 8.0), (2, 1, 512, 6, 512, 32, 1.0)])
def test_rotate_rms_append(ops, cuda, dtype, Hq, Hkv, dim, rot, pad, page, factor):
    g = gen(dim)
    pos = [0, 1, 15, 16, 33, 500, -1]
    T = len(pos)
    x = torch.randn(T, (Hq + Hkv) * dim + 5, generator=g).to(dtype)
    bias = torch.randn((Hq + Hkv) * dim, generator=g)
    bt, n_pages = _table(g, 2, 40, cuda)
    slot = [1, 0, 1, 0, 1, 0, 1]
    K, V = (torch.full((n_pages, Hkv, page, pad), float("nan"), dtype=dtype, device=cuda) for _ in range(2))
    q = torch.full((T, Hq * pad), float("nan"), dtype=dtype, device=cuda)
    freq = torch.tensor([900.0 ** (-2.0 * i / max(rot, 1)) / factor for i in range(rot // 2)], dtype=torch.float64)
    ops.rotate_rms_append(x.to(cuda), bias.to(cuda), freq.float().to(cuda), rot, dim, 1e-3, 0.3, q, K, V, bt, i32(slot, cuda),
                          i32(pos, cuda), Hq, Hkv)
    xb = (x[:, :(Hq + Hkv) * dim].double() + bias.double()).view(T, Hq + Hkv, dim)
    y = orl.rms(orl.rotate(xb, torch.tensor(pos), rot, 900.0, factor), 1e-3)
    for t in range(T - 1):
        close(q[t].view(Hq, pad)[:, :dim], y[t, :Hq] * 0.3, dtype, bf=5e-3, f32=1e-4)
        page_id = int(bt[slot[t], pos[t] // page])
        close(K[page_id, :, pos[t] % page, :dim], y[t, Hq:], dtype, bf=5e-3, f32=1e-4)
        close(V[page_id, :, pos[t] % page, :dim], xb[t, Hq:], dtype, bf=5e-3)
        assert not K[page_id, :, pos[t] % page, dim:].any() and not V[page_id, :, pos[t] % page, dim:].any()
    assert not q[:-1].view(-1, pad)[:, dim:].any()
    assert int((~K.isnan()).any(-1).sum()) == (T - 1) * Hkv  # nothing else, and nothing for the padding row


# ---------------------------------------------------------------- attention: chunks, sinks, heads that share keys
def _attention_case(cuda, dtype, n, Hq, Hkv, D, page, seed, far):
    """Random heads in which chosen (query, key) pairs have a score that decides the row.  ``far``: list of such pairs."""
    g = gen(seed)
    q, k, v = (torch.randn(n, h, D, generator=g).to(dtype) for h in (Hq, Hkv, Hkv))
    q, k = q * D ** -0.5, k
    for i, j in far:
        q[i] = k[j].repeat_interleave(Hq // Hkv, 0) * (12.0 / D)  # score 12 on average, the others +-1
    bt, n_pages = _table(g, 1, -(-n // page), cuda)
    K, V = (torch.full((n_pages, Hkv, page, D), float("nan"), dtype=dtype, device=cuda) for _ in range(2))
    for j in range(n):
        K[int(bt[0, j // page]), :, j % page], V[int(bt[0, j // page]), :, j % page] = k[j].to(cuda), v[j].to(cuda)
    return q, k, v, bt, K, V, torch.randn(Hq, generator=g) * 2 + 2


def _attention_want(q, k, v, chunk, sink, scale):
    rep = q.shape[1] // k.shape[1]
    kk, vv = k.double().repeat_interleave(rep, 1), v.double().repeat_interleave(rep, 1)
    s = torch.einsum("ihd,jhd->hij", q.double(), kk) * scale
    s = s.masked_fill(~orl.chunk_mask(q.shape[0], chunk or None), float("-inf"))
    w = orl.sink_softmax(s, sink.double()) if sink is not None else torch.softmax(s, -1)
    return torch.einsum("hij,jhd->ihd", w, vv)


@pytest.mark.parametrize("Hq,Hkv,D,page,chunk,n", [(4, 2, 64, 16, 23, 150), (6, 1, 128, 16, 100, 330), (3, 3, 64, 32, 64, 200), (2, 2, 128, 32, 0, 300),
                                                   (2, 1, 64, 16, 7, 140), (1, 1, 128, 16, 256, 520), (8, 2, 64, 32, 129, 400)])
def test_chunked_attention_with_sinks(ops, cuda, Hq, Hkv, D, page, chunk, n):
    """Prompt rows (from different starts), single rows, splits of a row's keys: just inside and just outside a chunk's edge, the
    chunk's first key, page borders.  A query that asks for a key outside must not get it."""
    c = chunk or n
    edges = [(c, c - 1), (c, c), (c + 5, c + 1), (2 * c - 1, c), (2 * c - 1, c - 1), (c + 2, 0), (n - 1, (n - 1) // c * c), (page, page - 1), (33, 16), (40, 0)]
    far = [(i, j) for i, j in edges if 0 <= j <= i < n]
    q, k, v, bt, K, V, sink = _attention_case(cuda, BF, n, Hq, Hkv, D, page, n + D, far)
    for sk in (sink, None):
        want = _attention_want(q, k, v, chunk, sk, 0.9)
        dsk = sk.to(cuda) if sk is not None else None
        qd = q.reshape(n, -1).to(cuda)
        kw = dict(chunk=chunk, sink=dsk)
        slot, status = torch.zeros(n, dtype=torch.int32, device=cuda), torch.zeros(1, dtype=torch.int32, device=cuda)
        for first in (0, 1, c - 1, c, c + 3):
            if first >= n:
                continue
            tiles = i32([(0, r, min(128, n - first - r), first + r) for r in range(0, n - first, 128)], cuda)
            out = torch.full((n - first, Hq * D), float("nan"), dtype=BF, device=cuda)
            ops.prefill_attention_masked(qd[first:], K, V, bt, tiles, len(tiles), Hq, 0.9, out, status=status, **kw)
            close(out.view(-1, Hq, D), want[first:], BF)
        assert not status.any()
        pos = i32(range(n), cuda)
        for splits in (1, 3):
            work = torch.zeros(max(ops.paged_attention_workspace(n, Hq, D, splits), 16), dtype=torch.uint8, device=cuda)
            out = torch.full((n, Hq * D), float("nan"), dtype=BF, device=cuda)
            ops.paged_attention_masked(qd, K, V, bt, slot, pos, Hq, 0.9, out, n_splits=splits, work=work, **kw)
            close(out.view(n, Hq, D), want, BF)


@pytest.mark.parametrize("Hq,Hkv,dim,rot,pad,page,chunk", [(4, 2, 36, 20, 64, 16, 23), (5, 1, 72, 72, 128, 32, 40), (8, 2, 128, 64, 128, 16, 0),
                                                           (2, 2, 64, 0, 64, 32, 64), (1, 1, 64, 64, 64, 16, 7)])
@pytest.mark.parametrize("splits", [1, 4])
def test_decode_attention_in_one_launch(ops, cuda, Hq, Hkv, dim, rot, pad, page, chunk, splits):
    """Token by token: rotation, norm, append and attention in one launch against the oracle over the whole sequence."""
    n, g = 90, gen(dim + chunk)
    x = torch.randn(n, (Hq + Hkv) * dim, generator=g).to(BF)
    bias, sink = torch.randn((Hq + Hkv) * dim, generator=g), torch.randn(Hq, generator=g) + 2
    freq = torch.tensor([500.0 ** (-2.0 * i / max(rot, 1)) / 2.0 for i in range(rot // 2)], dtype=torch.float64)
    bt, n_pages = _table(g, 2, 10, cuda)
    K, V = (torch.full((n_pages, Hkv, page, pad), float("nan"), dtype=BF, device=cuda) for _ in range(2))
    scale = 3.0 / dim ** 0.5
    work = torch.zeros(max(ops.paged_attention_workspace(2, Hq, pad, splits), 16), dtype=torch.uint8, device=cuda)
    got = []
    for t in range(n):  # (a second row is padding: it stores nothing)
        out = torch.full((2, Hq * pad), float("nan"), dtype=BF, device=cuda)
        ops.paged_attention_rms(x[[t, t]].to(cuda), bias.to(cuda), freq.float().to(cuda), rot, dim, 1e-3, K, V, bt, i32([1, 0], cuda),
                                i32([t, -1], cuda), Hq, scale, out, chunk=chunk, sink=sink.to(cuda), n_splits=splits, work=work)
        got.append(out[0].view(Hq, pad))
    assert not torch.stack(got)[..., dim:].any()
    xb = (x.double() + bias.double()).view(n, Hq + Hkv, dim)
    y = orl.rms(orl.rotate(xb, torch.arange(n), rot, 500.0, 2.0), 1e-3)
    close(torch.stack(got)[..., :dim], _attention_want(y[:, :Hq], y[:, Hq:], xb[:, Hq:], chunk, sink, scale), BF)
    assert K[bt[0].long()].isnan().all()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("Hq,Hkv,D,page,chunk,n", [(4, 2, 40, 16, 23, 90), (2, 1, 144, 32, 70, 150), (1, 1, 512, 16, 0, 40), (3, 3, 8, 16, 5, 60)])
def test_plain_attention_kernel(ops, cuda, dtype, Hq, Hkv, D, page, chunk, n):
    c = chunk or n
    far = [(i, j) for i, j in [(c, c - 1), (c, c), (c + 2, c), (2 * c - 1, c), (2 * c - 1, c - 1), (20, 16), (20, 0)] if 0 <= j <= i < n]
    q, k, v, bt, K, V, sink = _attention_case(cuda, dtype, n, Hq, Hkv, D, page, n + D, far)
    out = torch.full((n + 1, Hq * D), float("nan"), dtype=dtype, device=cuda)
    qd = torch.cat([q.reshape(n, -1), q[:1].reshape(1, -1)]).to(cuda)
    slot, pos = torch.zeros(n + 1, dtype=torch.int32, device=cuda), i32(list(range(n)) + [-1], cuda)
    ops.paged_attention_masked(qd, K, V, bt, slot, pos, Hq, -0.8, out, chunk=chunk, sink=sink.to(cuda))
    close(out[:n].view(n, Hq, D), _attention_want(q, k, v, chunk, sink, -0.8), dtype)
    ops.paged_attention_masked(qd, K, V, bt, slot, pos, Hq, 0.8, out, chunk=chunk)
    close(out[:n].view(n, Hq, D), _attention_want(q, k, v, chunk, None, 0.8), dtype)
    assert not out[n].any()


# ---------------------------------------------------------------- gated delta rule
class DeltaCase:
    """One delta layer between projection and output norm: projected rows of several sequences, and what the oracle makes of
    each (outputs after norm and gate, state)."""

    def __init__(self, ops, cuda, dtype, heads, kv, dim, vdim, taps, lengths, seed=0):
        g = gen(seed + dim)
        up = lambda n: -(-n // 8) * 8
        dk, dv, hp = up(dim), up(vdim), up(heads)
        self.dk, self.dv, self.dim, self.vdim, self.heads, self.dtype, self.cuda, self.ops = dk, dv, dim, vdim, heads, dtype, cuda, ops
        conv = 0.3 + 0.5 * torch.randn(2 * kv * dim + heads * vdim, taps, generator=g)
        A_log, dt, w = torch.rand(heads, generator=g) * 4 - 4, torch.rand(heads, generator=g) * 2 - 3, 1 + 0.2 * torch.randn(vdim, generator=g)
        spread = lambda t, n, d, p: torch.nn.functional.pad(t.reshape(*t.shape[:-1], n, d), (0, p - d)).flatten(-2)
        cut = [kv * dim, kv * dim, heads * vdim]
        lay = lambda t: torch.cat([spread(x, n, d, p) for x, n, d, p in zip(t.split(cut, -1), (kv, kv, heads), (dim, dim, vdim), (dk, dk, dv))], -1)
        C = 2 * kv * dk + heads * dv
        self.rule = ops.DeltaRule(heads, kv, dk, dv, vdim, taps, dim ** -0.5, C, C + heads * dv, C + heads * dv + hp,
                                  lay(conv.t().contiguous()).contiguous().to(cuda), A_log.to(cuda), dt.to(cuda),
                                  torch.nn.functional.pad(w, (0, dv - vdim)).to(cuda))
        self.rows, self.want, self.want_state = [], [], []
        D = lambda t: t.double()
        for n in lengths:
            x = torch.randn(n, sum(cut), generator=g).to(dtype)
            if n > 8:  # a value written once under a key that is asked for much later
                x[2, :cut[0] + cut[1]] *= 4
                x[n - 2, :cut[0]] = x[2, cut[0]:cut[0] + cut[1]]
            gate, b, a = torch.randn(n, heads * vdim, generator=g).to(dtype), torch.randn(n, heads, generator=g).to(dtype), torch.randn(n, heads, generator=g).to(dtype)
            hpad = lambda t: torch.nn.functional.pad(t, (0, hp - heads))
            self.rows.append(torch.cat([lay(x), spread(gate, heads, vdim, dv), hpad(b), hpad(a)], -1))
            y = orl.silu(orl.short_conv(D(x), D(conv)))
            q, k, v = y.split(cut, -1)
            q, k = orl.unit(q.view(n, kv, dim)) * dim ** -0.5, orl.unit(k.view(n, kv, dim))
            dec, beta = orl.delta_decay(D(a), D(A_log), D(dt)), torch.sigmoid(D(b))
            per = [orl.delta_rule(q[:, h // (heads // kv)], k[:, h // (heads // kv)], v.view(n, heads, vdim)[:, h], dec[:, h], beta[:, h])
                   for h in range(heads)]
            o = torch.stack([p[0] for p in per], 1)
            self.want.append(orl.rms(o, 1e-4) * D(w) * orl.silu(D(gate)).view(n, heads, vdim))
            self.want_state.append(torch.stack([p[1] for p in per]))
        nan = float("nan")  # whatever a slot held before must not matter
        self.state = torch.full((len(lengths) + 2, heads, dk, dv), nan, device=cuda)
        self.ring = torch.full((len(lengths) + 2, taps, C), nan, dtype=dtype, device=cuda)
        self.at = [0] * len(lengths)
        self.got = [[] for _ in lengths]

    def slot(self, s):
        return len(self.rows) - s

    def scan(self, parts, chunks=False):
        """parts: (sequence, rows) in the order of the pass.  chunks: 64 tokens at a time on the tensor cores."""
        ops, r, cuda = self.ops, self.rule, self.cuda
        segs, rows, slots, pos, first = [], [], [], [], 0
        for s, n in parts:
            segs.append((self.slot(s), first, n, self.at[s]))
            rows.append(self.rows[s][self.at[s]:self.at[s] + n])
            slots += [self.slot(s)] * n
            pos += range(self.at[s], self.at[s] + n)
            first += n
        x = torch.cat(rows).contiguous().to(cuda)
        T, nan = len(slots), float("nan")
        xc = torch.full((T, r.channels), nan, dtype=self.dtype, device=cuda)
        o = torch.full((T, r.heads * r.vdim), nan, device=cuda)
        out = torch.full((T, r.heads * r.vdim), nan, dtype=self.dtype, device=cuda)
        ops.short_conv(x, r.conv, self.ring, i32(slots, cuda), i32(pos, cuda), xc)
        if chunks:
            work = torch.full((ops.delta_chunk_workspace(T, len(segs), r.heads),), 255, dtype=torch.uint8, device=cuda)
            status = torch.zeros(1, dtype=torch.int32, device=cuda)
            ops.delta_chunk(xc, x, r, i32(segs, cuda), len(segs), max(n for _, n in parts), self.state, self.ring, o, work, status)
            assert not int(status)
        else:
            ops.delta_scan(xc, x, r, i32(segs, cuda), len(segs), self.state, self.ring, o)
        self.raw = o
        ops.gated_rms(o, x[:, r.g_col:], r.norm, r.heads, r.vdim_true, 1e-4, out)
        for (s, n), (_, a, _, _) in zip(parts, segs):
            self.got[s].append(out[a:a + n])
            self.at[s] += n

    def step(self, seqs):
        """One token of each; -1: a padding row."""
        ops, r, cuda = self.ops, self.rule, self.cuda
        x = torch.stack([self.rows[max(s, 0)][min(self.at[max(s, 0)], len(self.rows[max(s, 0)]) - 1)] for s in seqs]).to(cuda)
        out = torch.full((len(seqs), r.heads * r.vdim), float("nan"), dtype=self.dtype, device=cuda)
        ops.delta_step(x, r, 1e-4, i32([self.slot(s) if s >= 0 else 0 for s in seqs], cuda), i32([self.at[s] if s >= 0 else -1 for s in seqs], cuda),
                       self.state, self.ring, out)
        for i, s in enumerate(seqs):
            if s >= 0:
                self.got[s].append(out[i:i + 1])
                self.at[s] += 1
            else:
                assert not out[i].any()

    def check(self, f32=1e-4, bf=3e-2):
        for s, want in enumerate(self.want):
            got = torch.cat(self.got[s]).view(-1, self.heads, self.dv).cpu()
            assert not got[..., self.vdim:].any()
            close(got[..., :self.vdim], want[:len(got)], self.dtype, bf=bf, f32=f32)
            if len(got) == len(want):
                S = self.state[self.slot(s)].cpu()
                close(S[:, :self.dim, :self.vdim], self.want_state[s], self.dtype, bf=bf, f32=f32)
                assert not S[:, self.dim:].any() and not S[..., self.vdim:].any()
        assert self.state[-1].isnan().all() and self.state[0].isnan().all()  # other slots untouched


SIZES = [(6, 2, 20, 12, 3), (3, 3, 33, 41, 5), (1, 1, 8, 8, 1), (2, 1, 200, 8, 2), (4, 4, 128, 136, 4), (2, 2, 64, 64, 8), (2, 1, 96, 264, 4), (3, 1, 256, 48, 6), (1, 1, 256, 208, 3)]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("size", SIZES)
def test_delta_whole_sequences(ops, cuda, dtype, size):
    c = DeltaCase(ops, cuda, dtype, *size, lengths=(1, 40, 2, 17, 130))
    c.scan([(1, 40), (0, 1), (4, 130), (2, 2), (3, 17)])
    c.check()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("size", SIZES)
def test_delta_portions_and_single_tokens(ops, cuda, dtype, size):
    """Portions down to one and two tokens (shorter than the convolution), then decoded tokens, then a portion again."""
    c = DeltaCase(ops, cuda, dtype, *size, lengths=(60, 33))
    for part in ([(0, 1)], [(0, 2), (1, 20)], [(1, 2), (0, 2)], [(0, 17)], [(0, 1), (1, 1)]):
        c.scan(part)
    for _ in range(6):
        c.step([1, -1, 0])
    c.scan([(0, 20), (1, 2)])
    while c.at[0] < 60:
        c.step([0])
    c.scan([(1, 2)])
    c.check()


CHUNKED = [(2, 2, 64, 64, 4), (4, 2, 64, 24, 3), (3, 1, 128, 128, 4), (2, 2, 128, 200, 2), (1, 1, 57, 33, 4), (2, 1, 121, 136, 5)]


@pytest.mark.parametrize("size", CHUNKED)
def test_delta_chunks_whole_sequences(ops, cuda, size):
    c = DeltaCase(ops, cuda, BF, *size, lengths=(1, 64, 2, 63, 200, 65, 128))
    c.scan([(1, 64), (0, 1), (4, 200), (2, 2), (3, 63), (6, 128), (5, 65)], chunks=True)
    c.check()
    # the same rows one token at a time: equal to fp32 rounding, before anything is rounded to 16 bits
    one = DeltaCase(ops, cuda, BF, *size, lengths=(1, 64, 2, 63, 200, 65, 128))
    one.scan([(1, 64), (0, 1), (4, 200), (2, 2), (3, 63), (6, 128), (5, 65)])
    close(c.raw, one.raw, F32, f32=5e-6)
    used = slice(1, len(c.rows) + 1)
    close(c.state[used], one.state[used], F32, f32=5e-6)
    assert torch.equal(c.ring.nan_to_num(), one.ring.nan_to_num())


@pytest.mark.parametrize("size", CHUNKED[:4])
def test_delta_chunks_portions_and_single_tokens(ops, cuda, size):
    c = DeltaCase(ops, cuda, BF, *size, lengths=(300, 150))
    for part in ([(0, 1)], [(0, 2), (1, 20)], [(1, 70), (0, 64)], [(0, 100)], [(1, 1), (0, 65)]):
        c.scan(part, chunks=True)
    for _ in range(6):
        c.step([1, -1, 0])
    c.scan([(0, 20), (1, 2)])
    c.scan([(0, 40), (1, 50)], chunks=True)
    while c.at[1] < 150:
        c.step([1])
    c.scan([(0, 2)], chunks=True)
    c.check()


def test_delta_chunks_many_tokens_and_strong_decays(ops, cuda):
    """Long walks; decays from almost none to complete within a few tokens."""
    for shift in (0.0, 4.0, 8.0):
        c = DeltaCase(ops, cuda, BF, 2, 1, 64, 32, 4, lengths=(1500,))
        c.rule.A_log += shift
        one = DeltaCase(ops, cuda, BF, 2, 1, 64, 32, 4, lengths=(1500,))
        one.rule.A_log += shift
        c.scan([(0, 1500)], chunks=True)
        one.scan([(0, 1500)])
        close(c.raw, one.raw, F32, f32=2e-5)
        close(c.state[1], one.state[1], F32, f32=2e-5)


def test_delta_many_tokens_one_by_one(ops, cuda):
    c = DeltaCase(ops, cuda, F32, 2, 1, 24, 16, 4, lengths=(300,))
    while c.at[0] < 300:
        c.step([0])
    c.check()


@pytest.mark.parametrize("n_seq", [1, 9, 40])
def test_delta_column_parts(ops, cuda, n_seq):
    """However many CTAs share a head's columns, the bits are the same."""
    c = DeltaCase(ops, cuda, F32, 8, 8, 128, 128, 4, lengths=[11] * n_seq)
    c.scan([(s, 11) for s in range(n_seq)])
    c.check()
    one = DeltaCase(ops, cuda, F32, 8, 8, 128, 128, 4, lengths=[11] * n_seq)
    one.scan([(n_seq - 1, 11)])
    assert torch.equal(one.got[n_seq - 1][0], c.got[n_seq - 1][0])


def test_host_checks(ops, cuda):
    z = torch.zeros(64, 64, device=cuda)
    e = load("_lib").MloraError
    with pytest.raises(e, match="streams"):
        ops.residual_streams_layernorm(None, z, torch.ones(17, device=cuda), z[0].bfloat16(), 1e-5, 64, z.clone())
    with pytest.raises(e, match="taps"):
        ops.short_conv(z, torch.zeros(9, 64, device=cuda), z, i32([0] * 64, cuda), i32([0] * 64, cuda), z.clone())
    with pytest.raises(e, match="dim"):
        DeltaCase(ops, cuda, F32, 1, 1, 264, 8, 2, lengths=(2,)).scan([(0, 2)])
