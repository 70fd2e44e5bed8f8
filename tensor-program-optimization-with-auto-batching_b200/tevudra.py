"""Tevudra: pre-norm decoder with latent attention, dense or mixture-of-experts feed-forward layers and dynamic tanh norms.

Per layer (h = dyt(x), the residual x in fp32):

    [q | latent | gates] = W_in h                       one projection (layers that read another layer's latents: [q | gates])
    c = rms(latent)  -> page                            ``PagedLatentCache``; layers with ``kv_from`` use that layer's pages
    decode, short portions:  qa_h = W_uk_h^T q_h;  s = softmax(scale qa_h . c_j) c_j;  o_h = (W_uv_h s) sigmoid(gate_h)
    prompt passes:           [k | v] = [W_uk; W_uv] c for the whole context, causal attention on the tensor cores, gated
    x += W_o o
    x += W_down relu^2(W_up h)   or   sum over the chosen experts and the shared one of w_e W_down_e gelu(W_up_e h)

Each mechanism is a kernel of its own with sizes and constants as arguments; this file only lays weights out and orders the
launches.  ``dtype`` bfloat16: tensor-core projections and attention; float32: the same sequence on true 32-bit kernels.
Sizes need no alignment: weights are zero-padded at load (rows of activations to multiples of 8, heads to 64s).
"""
from __future__ import annotations

from dataclasses import dataclass

import numpy as np
import torch

from . import ops
from .engine import PlainEngine
from .kv_cache import PagedLatentCache
from .ops import ACT_GELU, ACT_RELU2, OUT_F32
from .packing import PackedDesign, up as _up


def _head_pad(d):
    """Head sizes the tensor-core attention takes: 64 and 128; larger heads only run in latent space."""
    return _up(d, 64)


@dataclass(frozen=True)
class LatentAttention:
    heads: int
    dim: int
    vdim: int
    rank: int
    scale: float
    source: int  # layer whose latents are read (its own index: computes them)


@dataclass(frozen=True)
class Dense:
    ff: int


@dataclass(frozen=True)
class MoE:
    ff: int
    experts: int
    top: int
    shared_ff: int  # 0: no shared expert


@dataclass(frozen=True)
class TevudraConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple  # of (LatentAttention, Dense | MoE | None)

    @classmethod
    def parse(cls, cfg):
        """The ``config.json`` of a checkpoint (a dict)."""
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            if entry["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
            m = entry["mixer"]
            mix = LatentAttention(m["heads"], m["dim"], m["vdim"], m["kv_rank"], float(m["scale"]), m.get("kv_from", i))
            if mix.source != i:
                if not 0 <= mix.source < i or layers[mix.source][0].source != mix.source:
                    raise ValueError(f"layer {i}: kv_from {mix.source} names no earlier layer with latents of its own")
                if layers[mix.source][0].rank != mix.rank:
                    raise ValueError(f"layer {i}: kv_rank differs from that of layer {mix.source}")
            f = entry.get("mlp")
            if f is None:
                ff = None
            elif f["kind"] == "dense":
                ff = Dense(f["ff"])
            elif f["kind"] == "moe":
                ff = MoE(f["expert"]["ff"], f["router"]["experts"], f["router"]["top"], (f.get("shared") or {"ff": 0})["ff"])
                if not 1 <= ff.top <= ff.experts:
                    raise ValueError(f"layer {i}: top {ff.top} of {ff.experts} experts")
            else:
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            layers.append((mix, ff))
        return cls(cfg["vocab"], cfg["width"], float(cfg["norm"]["eps"]), tuple(layers))


class _Norm:
    def __init__(self, get, name, width, device):
        vec = lambda t: torch.nn.functional.pad(t.to(device, torch.bfloat16).reshape(-1), (0, width - t.numel())).contiguous()
        self.w, self.b = vec(get(name)), vec(get(name + ".b"))
        self.alpha = get(name + ".alpha").to(device, torch.bfloat16).reshape(1)


class _Layer:
    """Packed weights of one layer."""


class PackedTevudra(PackedDesign):
    """Device-resident weights.  ``weights``: tensors under the checkpoint's names (``embed``, ``l<i>.mix.q``, ...)."""

    name = "Tevudra"

    def __init__(self, cfg, weights, device="cuda", dtype=torch.bfloat16):
        self.config = c = TevudraConfig.parse(cfg)
        super().__init__(cfg, c.vocab, c.width, len(c.layers), device, dtype)
        get = lambda n: weights[n]
        self.embed = self._mat(get("embed"), (c.vocab, self.H), torch.bfloat16)
        self.norm = _Norm(get, "final.norm", self.H, self.device)
        self.head = self._weight(get("head"), (c.vocab, self.H))
        self.layers = [self._layer(i, mix, ff, get) for i, (mix, ff) in enumerate(c.layers)]

    def _layer(self, i, mix, ff, get):
        lw, H, dev = _Layer(), self.H, self.device
        p = f"l{i}.mix."
        lw.mix, lw.ff = mix, ff
        lw.norm1 = _Norm(get, f"l{i}.norm1", H, dev)
        lw.dk, lw.dv, lw.rq = _head_pad(mix.dim), _head_pad(mix.vdim), _up(mix.rank, 128)
        heads = lambda t, d, pad: self._mat(t.reshape(mix.heads, d, -1), (mix.heads, pad, t.shape[-1]))
        q = heads(get(p + "q"), mix.dim, lw.dk).flatten(0, 1)
        parts = [self._mat(q, (q.shape[0], H))]
        lw.c_col = q.shape[0]
        own = mix.source == i
        if own:
            parts.append(self._mat(get(p + "dkv"), (_up(mix.rank, 8), H)))
            lw.c_norm = get(p + "dkv.norm").to(dev, torch.bfloat16).contiguous()
        lw.g_col = sum(t.shape[0] for t in parts)
        parts.append(self._mat(get(p + "g"), (_up(mix.heads, 8), H)))
        w_in = torch.cat(parts)
        lw.w_in = self._weight(w_in, tuple(w_in.shape))
        lw.in_cols = w_in.shape[0]
        uk, uv = heads(get(p + "uk"), mix.dim, lw.dk), heads(get(p + "uv"), mix.vdim, lw.dv)  # [heads, d, rank]
        lw.absorb = ops.GroupedWeight(self._mat(uk.transpose(1, 2), (mix.heads, lw.rq, lw.dk)))
        lw.uv = ops.GroupedWeight(self._mat(uv, (mix.heads, lw.dv, lw.rq)))
        # keys and values of a whole context at once (prompt passes on the tensor cores)
        lw.expand = None
        if self.dtype == torch.bfloat16 and lw.dk <= 128 and lw.dv <= 128 and mix.scale > 0:
            ukv = torch.cat([uk.flatten(0, 1), uv.flatten(0, 1)])
            lw.expand = self._weight(ukv, (ukv.shape[0], _up(mix.rank, 64)))
        o = get(p + "o").reshape(self.width, mix.heads, mix.vdim)
        lw.w_o = self._weight(self._mat(o, (H, mix.heads, lw.dv)).flatten(1), (H, mix.heads * lw.dv))
        if ff is None:
            return lw
        p = f"l{i}.mlp."
        lw.norm2 = _Norm(get, f"l{i}.norm2", H, dev)
        if isinstance(ff, Dense):
            lw.ffp = _up(ff.ff, 8)
            lw.up, lw.down = self._weight(get(p + "up"), (lw.ffp, H)), self._weight(get(p + "down"), (H, lw.ffp))
            return lw
        lw.ffp = _up(ff.ff, 8)
        lw.router_rows = self._mat(get(p + "router"), (ff.experts, H))  # decode steps: routed in one launch
        lw.router = ops.GroupedWeight(lw.router_rows[None])
        lw.router_b = get(p + "router.b").to(dev, torch.float32).contiguous()
        stack = lambda n, shape: ops.GroupedWeight(torch.stack([self._mat(get(f"{p}e{e}.{n}"), shape) for e in range(ff.experts)]))
        lw.e_up, lw.e_down = stack("up", (lw.ffp, H)), stack("down", (H, lw.ffp))
        if ff.shared_ff:
            lw.sffp = _up(ff.shared_ff, 8)
            lw.s_up, lw.s_down = self._weight(get(p + "shared.up"), (lw.sffp, H)), self._weight(get(p + "shared.down"), (H, lw.sffp))
        return lw

    # -- what the model is served with ----------------------------------------------------------------------------
    def new_cache(self, max_batch, max_total_seq_len, prefill_chunk, page_size=16, max_seq_len=None):
        ranks = {i: lw.mix.rank for i, lw in enumerate(self.layers) if lw.mix.source == i}
        return PagedLatentCache(ranks, max_batch, max_total_seq_len, prefill_chunk, page_size, self.device,
                                max_seq_len=max_seq_len, dtype=self.dtype)

    def new_engine(self, kv, max_rows):
        return TevudraEngine(self, kv, max_rows)


class TevudraEngine(PlainEngine):
    # a prompt pass expands keys and values of at most this many context rows; beyond, its rows attend in latent space
    MAX_EXPANDED_ROWS = 1 << 18
    # cost of an operation in latent space (row by row) against one of the tiled prompt attention
    LATENT_COST = 3.0

    def __init__(self, model: PackedTevudra, kv: PagedLatentCache, max_rows: int):
        shapes = [(model.H, model.V)]
        for lw in model.layers:
            shapes += [(model.H, lw.in_cols), (lw.mix.heads * lw.dv, model.H)]
            if isinstance(lw.ff, Dense):
                shapes += [(model.H, lw.ffp), (lw.ffp, model.H)]
            elif lw.ff is not None:
                shapes += [(model.H, lw.sffp), (lw.sffp, model.H)] if lw.ff.shared_ff else []
        super().__init__(model, kv, max_rows, shapes, ops._lib.lib().mlora_grouped_linear_workspace(64))
        m, dev, T = model, model.device, self.max_rows
        act = dict(dtype=m.dtype, device=dev)
        lws, moes = m.layers, [lw for lw in m.layers if isinstance(lw.ff, MoE)]
        self.res = torch.zeros(T, m.H, dtype=torch.float32, device=dev)
        self.xn = torch.zeros(T, m.H, **act)
        self.y = torch.zeros(T, m.H, **act)
        widest = lambda f, ls: max([f(lw) for lw in ls], default=8)
        self.proj = torch.zeros(T * widest(lambda lw: lw.in_cols, lws), **act)
        self.attn = torch.zeros(T * widest(lambda lw: lw.mix.heads * lw.dv, lws), **act)
        hidden = [lw.ffp for lw in lws if isinstance(lw.ff, Dense)] + [lw.sffp for lw in moes if lw.ff.shared_ff]
        self.act = torch.zeros(T * max(hidden + [8]), **act)
        if moes:
            pairs = lambda lw: T * lw.ff.top
            self.plans = {}  # (experts, top) -> buffers of the routing
            for lw in moes:
                key = (lw.ff.experts, lw.ff.top)
                if key not in self.plans:
                    self.plans[key] = ops.MoePlan(T, *key, dev)
            self.router_out = torch.zeros(T * widest(lambda lw: lw.ff.experts, moes), dtype=torch.float32, device=dev)
            self.e_act = torch.zeros(widest(lambda lw: pairs(lw) * lw.ffp, moes), **act)
            self.e_out = torch.zeros(widest(lambda lw: pairs(lw) * m.H, moes), **act)
        # prompt passes: query tiles of <= 128 rows, context segments (whole pages) of the expanded keys and values
        self.tiles = torch.zeros((T + 127) // 128 + kv.max_batch + 1, 4, dtype=torch.int32, device=dev)
        self.segs = torch.zeros(kv.max_batch, 4, dtype=torch.int32, device=dev)
        self._n_tiles = self._n_segs = self._ctx_rows = self._max_ctx = 0

    # -- prompt passes ------------------------------------------------------------------------------------------
    def _begin_prompt_pass(self, chunk):
        """Expanded keys and values when that costs less than attending in latent space.  Per head and new row, latent
        space costs 4 R per key, expanded keys 2 (dk + dv), and expanding a context row costs 2 R (dk + dv)."""
        self._n_tiles = 0
        ps = self.kv.page_size
        ctx = [_up(p0 + n, ps) for _, _, n, p0 in chunk]
        if any(lw.expand is None for lw in self.m.layers) or sum(ctx) > self.MAX_EXPANDED_ROWS:
            return
        latent = expanded = 0
        pairs = sum(n * (p0 + n / 2) for _, _, n, p0 in chunk)
        for lw in self.m.layers:
            R, d = lw.mix.rank, lw.dk + lw.dv
            latent += lw.mix.heads * 4 * R * pairs
            expanded += lw.mix.heads * (2 * d * pairs + 2 * R * d * sum(ctx))
        if latent * self.LATENT_COST < expanded:
            return
        tiles, segs, base = [], [], 0
        for (sid, r0, n, p0), c in zip(chunk, ctx):
            segs.append((self.kv.slot(sid), base, p0 + n, 0))
            tiles += [(base, r0 + off, min(128, n - off), p0 + off) for off in range(0, n, 128)]
            base += c
        if len(tiles) > self.tiles.shape[0] or len(segs) > self.segs.shape[0]:
            return
        self._stage(self.tiles.view(-1), np.asarray(tiles, dtype=np.int32).reshape(-1), torch.int32)
        self._stage(self.segs.view(-1), np.asarray(segs, dtype=np.int32).reshape(-1), torch.int32)
        self._n_tiles, self._n_segs, self._ctx_rows, self._max_ctx = len(tiles), len(segs), base, max(ctx)

    def _end_prompt_pass(self):
        self._n_tiles = 0

    # -- pieces of a layer ----------------------------------------------------------------------------------------
    def _grouped(self, x, W, out, flags=0, **kw):
        if self.m.dtype == torch.float32:
            flags &= ~OUT_F32
        kw["flags"] = flags
        return ops.grouped_linear(x, W, out, work=self.ws_linear, **kw)

    def _attention(self, T, lw, fused_append):
        kv, mix, H = self.kv, lw.mix, lw.mix.heads
        row_slot, row_pos = self.row_slot[:T], self.row_pos[:T]
        proj = self._linear(self.xn[:T], lw.w_in, self.proj[:T * lw.in_cols].view(T, lw.in_cols))
        pages = kv.latent_pages(mix.source)
        if lw.g_col > lw.c_col:
            ops.latent_append(proj[:, lw.c_col:], mix.rank, lw.c_norm, self.m.config.eps, pages, kv.block_table, row_slot, row_pos)
        gate = proj[:, lw.g_col:]
        out = self.attn[:T * H * lw.dv].view(T, H * lw.dv)
        if not fused_append and self._n_tiles:
            S, R8, cols = self._ctx_rows, pages.shape[2], H * (lw.dk + lw.dv)
            c = ops.latent_gather(pages, kv.block_table, self.segs, self._n_segs, self._max_ctx, self._grow("ctx", S * R8).view(S, R8))
            ekv = self._linear(c, lw.expand, self._grow("ekv", S * cols).view(S, cols))
            ops.prefill_attention_dense(proj, ekv, H * lw.dk, self.tiles, self._n_tiles, H, lw.dk, lw.dv, mix.scale, out,
                                        gate=gate, status=self.status)
        else:
            tr = ops.grouped_tile_rows(T, self.m.dtype)
            qa = self._grow("qa", T * H * lw.rq).view(T, H * lw.rq)
            lat = self._grow("lat", T * H * lw.rq).view(T, H * lw.rq)
            self._grouped(proj, lw.absorb, qa, T=T, x_cols=lw.dk, y_cols=lw.rq, tile_rows=tr)
            splits, work = 1, None
            if self.m.dtype == torch.bfloat16 and mix.rank <= ops.LATENT_TC_MAX_RANK:
                splits = ops.latent_attention_splits(T, H, self.max_keys)
                nb = ops.latent_attention_workspace(T, H, lw.rq, splits)
                work = self._grow("merge", nb, torch.uint8) if nb else None
            ops.latent_attention(qa, mix.rank, H, pages, kv.block_table, row_slot, row_pos, mix.scale, lat, n_splits=splits,
                                 work=work, status=self.status)
            self._grouped(lat, lw.uv, out, T=T, x_cols=lw.rq, y_cols=lw.dv, tile_rows=tr, gate=gate)
        return self._linear(out, lw.w_o, self.y[:T])

    def _feed_forward(self, T, lw):
        """(rows to add to the residual or None, expert rows or None, their plan)."""
        m, ff, xn, y = self.m, lw.ff, self.xn[:T], self.y[:T]
        if isinstance(ff, Dense):
            a = self._linear(xn, lw.up, self.act[:T * lw.ffp].view(T, lw.ffp), ACT_RELU2)
            return self._linear(a, lw.down, y), None, None
        plan, n = self.plans[ff.experts, ff.top], T * ff.top
        tr = ops.grouped_tile_rows(n / ff.experts, m.dtype)
        if ops.moe_decode_fits(T, ff.top):
            ops.moe_route_plan(xn, lw.router_rows, lw.router_b, plan, tr)
        else:
            # few outputs, many rows: 64-row tiles fill the grid where the plain projection's larger ones do not
            logits = self._grouped(xn, lw.router, self.router_out[:T * ff.experts].view(T, ff.experts), T=T, tile_rows=64, flags=OUT_F32)
            ops.moe_plan(logits, lw.router_b, plan, T, tr)
        x, gather = xn, True
        if m.dtype == torch.bfloat16 and tr >= 128:
            # large tiles: rows copied into expert order first (four-row gathers cannot keep up with the tensor cores)
            x, gather = ops.embed(plan.rows[:n], xn, out_bf16=self._grow("e_in", n * m.H).view(n, m.H)), False
        a = self._grouped(x, lw.e_up, self.e_act[:n * lw.ffp].view(n, lw.ffp), plan=plan, gather=gather, flags=ACT_GELU)
        e = self._grouped(a, lw.e_down, self.e_out[:n * m.H].view(n, m.H), plan=plan)
        if not ff.shared_ff:
            return None, e, plan
        a = self._linear(xn, lw.s_up, self.act[:T * lw.sffp].view(T, lw.sffp), ACT_GELU)
        return self._linear(a, lw.s_down, y), e, plan

    def _norm(self, w, T, add, rows=None):
        """Adds what the layer before left (``add``) to the residual and normalises it into ``xn``."""
        delta, experts, plan = add
        n = T if rows is None else rows.numel()
        ops.residual_dyt(delta, self.res[:T], w.w, w.b, w.alpha, self.xn[:n], expert_rows=experts, plan=plan, rows=rows)

    def forward(self, T, fused_append, use_lora=True, lm_rows=None, n_lm=None, hidden=None):
        """One pass over the T rows staged in ``tokens`` / ``row_slot`` / ``row_pos``; as :meth:`model.Engine.forward`.
        (``use_lora`` and the staged adapter slots mean nothing to a design without adapters.)"""
        m = self.m
        if hidden is None:
            ops.embed(self.tokens[:T], m.embed, res=self.res[:T])
        else:
            ops.embed(self.iota[:T], hidden, res=self.res[:T])
        add = (None, None, None)
        for lw in m.layers:
            self._norm(lw.norm1, T, add)
            add = (self._attention(T, lw, fused_append), None, None)
            if lw.ff is not None:
                self._norm(lw.norm2, T, add)
                add = self._feed_forward(T, lw)
        rows = None if lm_rows is None else lm_rows[:n_lm]
        n = T if rows is None else n_lm
        self._norm(m.norm, T, add, rows)
        self._linear(self.xn[:n], m.head, self.logits[:n], OUT_F32)
        ops.argmax(self.logits[:n], out=self.next_tok[:n])
        return self.logits[:n], self.next_tok[:n]
