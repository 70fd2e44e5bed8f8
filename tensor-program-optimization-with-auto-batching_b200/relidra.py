"""Relidra: pre-norm decoder whose residual is several streams (hyper-connections), with gated delta-rule layers and chunked
attention layers, layer norms, dense feed-forwards and a run of layers that is passed through several times.

Per sublayer, with h = the layer norm of the streams' sum weighted by ``hc.in``:

    delta:      [q | k | v | gates | b | a] = W_in h                  one projection
                q, k, v = silu(short convolution over time)           inputs of the last tokens in a ring per sequence
                M' = c M + k w^T, w = step (v - c M^T k); o = M'^T q   state per head and sequence, fp32 (``HybridCache``)
                y = W_o (rms(o) w silu(gates))
    attention:  [q | k] = W_in h + bias;  v = k                       one projection
                q, k = rms(rotate(q)), rms(rotate(k)) -> page         rotation of part of a head
                y = W_o softmax over the row's own chunk, with a sink per head
    dense:      y = W_down gelu(W_up h)
    streams:    stream t' = y out_t + the old streams weighted by column t of ``hc.mix``

Each mechanism is a kernel of its own with sizes and constants as arguments; this file only lays weights out and orders the
launches.  ``dtype`` bfloat16: tensor-core projections and attention; float32: the same sequence on true 32-bit kernels.
Sizes need no alignment: weights are zero-padded at load (heads of delta layers to multiples of 8, of attention layers to 64
or 128).  A layer that runs several times has an entry in the cache for every run.
"""
from __future__ import annotations

from dataclasses import dataclass

import numpy as np
import torch

from . import ops
from .engine import PlainEngine
from .kv_cache import HybridCache
from .ops import ACT_GELU, OUT_F32
from .packing import PackedDesign, up


@dataclass(frozen=True)
class Delta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class Attention:
    heads: int
    kv_heads: int
    dim: int
    rot: int         # rotated columns of a head
    base: float
    factor: float    # every frequency is divided by it
    scale: float
    chunk: int       # positions a row sees lie in its own chunk of this many; 0: all before it


@dataclass(frozen=True)
class RelidraConfig:
    vocab: int
    width: int
    eps: float
    streams: int
    layers: tuple  # of (Delta | Attention, ff size or None)
    runs: tuple    # layer indices in the order they run

    @classmethod
    def parse(cls, cfg):
        """The ``config.json`` of a checkpoint (a dict)."""
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            m = entry["mixer"]
            if entry["type"] == "delta":
                mix = Delta(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
            elif entry["type"] == "attention":
                rot = m.get("rot") or {"dims": 0, "base": 1.0}
                mix = Attention(m["heads"], m["kv_heads"], m["dim"], rot["dims"], float(rot["base"]),
                                float((rot.get("scaling") or {"factor": 1.0})["factor"]), float(m["scale"]),
                                int((m.get("mask") or {"size": 0})["size"]))
                if m.get("vdim", mix.dim) != mix.dim:
                    raise ValueError(f"layer {i}: the values are the keys, but vdim {m['vdim']} is not dim {mix.dim}")
                if mix.rot % 2 or mix.rot > mix.dim:
                    raise ValueError(f"layer {i}: {mix.rot} rotated columns of a head of {mix.dim}")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
            if mix.kv_heads < 1 or mix.heads % mix.kv_heads:
                raise ValueError(f"layer {i}: {mix.heads} heads do not share {mix.kv_heads} kv_heads evenly")
            f = entry.get("mlp")
            if f is not None and f["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            layers.append((mix, f["ff"] if f else None))
        n, loop = len(layers), cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
        a, b = loop["start"], loop["stop"]
        if not (0 <= a <= b <= n and loop["times"] >= 0):
            raise ValueError(f"loop {loop} does not fit {n} layers")
        runs = list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))
        if cfg["streams"] < 1:
            raise ValueError("streams must be at least 1")
        return cls(cfg["vocab"], cfg["width"], float(cfg["norm"]["eps"]), cfg["streams"], tuple(layers), tuple(runs))


class _Layer:
    """Packed weights of one layer."""


class _Connection:
    """Coefficients of a sublayer: ``read`` = weights of its input's sum, ``back`` = what the streams get, then the mix."""

    def __init__(self, get, name, device):
        f = lambda n: get(f"{name}.{n}").to(device, torch.float32).reshape(-1)
        self.read, self.back = f("in").contiguous(), torch.cat([f("out"), f("mix")])


class PackedRelidra(PackedDesign):
    """Device-resident weights.  ``weights``: tensors under the checkpoint's names (``embed``, ``l<i>.mix.q``, ...)."""

    name = "Relidra"

    def __init__(self, cfg, weights, device="cuda", dtype=torch.bfloat16):
        self.config = c = RelidraConfig.parse(cfg)
        super().__init__(cfg, c.vocab, c.width, len(c.layers), device, dtype)
        get = lambda n: weights[n]
        self.embed = self._mat(get("embed"), (c.vocab, self.H), torch.bfloat16)
        self.head = self._weight(get("embed"), (c.vocab, self.H))
        self.norm = self._norm_weight(get("final.norm"))
        self.sum_streams = torch.ones(c.streams, dtype=torch.float32, device=self.device)
        self.layers = [self._layer(i, mix, ff, get) for i, (mix, ff) in enumerate(c.layers)]

    def _norm_weight(self, t):
        return self._mat(t, (self.H,), torch.bfloat16)

    def _f32(self, t, n):
        return self._mat(t.reshape(-1), (n,), torch.float32)

    def _layer(self, i, mix, ff, get):
        lw, p = _Layer(), f"l{i}."
        lw.mix = mix
        lw.norm1, lw.hc1 = self._norm_weight(get(p + "norm1")), _Connection(get, p + "hc1", self.device)
        (self._pack_delta if isinstance(mix, Delta) else self._pack_attention)(lw, mix, lambda n: get(p + "mix." + n))
        lw.ffp = 0
        if ff is not None:
            lw.norm2, lw.hc2 = self._norm_weight(get(p + "norm2")), _Connection(get, p + "hc2", self.device)
            lw.ffp = up(ff, 8)
            lw.up = self._weight(get(p + "mlp.up"), (lw.ffp, self.H))
            lw.down = self._weight(get(p + "mlp.down"), (self.H, lw.ffp))
        return lw

    def _in_weight(self, parts):
        """Weights with a common input as one projection, every part's rows padded to a multiple of 8."""
        w, cols, at = [], [], 0
        for t in parts:
            cols.append(at)
            w.append(self._mat(t, (up(t.shape[0], 8), self.H)))
            at += w[-1].shape[0]
        w = torch.cat(w)
        return self._weight(w, tuple(w.shape)), cols, at

    def _heads(self, t, heads, d, pad):
        """Rows of ``t`` [heads * d, ...] with every head padded to ``pad`` rows."""
        t = t.reshape(heads, d, -1)
        return self._mat(t, (heads, pad, t.shape[-1]), torch.float32).flatten(0, 1)

    def _pack_delta(self, lw, mix, get):
        dk, dv = up(mix.dim, 8), up(mix.vdim, 8)
        qk = lambda n: self._heads(get(n), mix.kv_heads, mix.dim, dk)
        v = lambda n: self._heads(get(n), mix.heads, mix.vdim, dv)
        lw.w_in, cols, lw.in_cols = self._in_weight([qk("q"), qk("k"), v("v"), v("g"), get("b"), get("a")])
        conv = torch.cat([qk("q.conv"), qk("k.conv"), v("v.conv")])
        if conv.shape[1] != mix.taps:
            raise ValueError(f"convolutions of {conv.shape[1]} taps, {mix.taps} in the configuration")
        lw.rule = ops.DeltaRule(mix.heads, mix.kv_heads, dk, dv, mix.vdim, mix.taps, mix.dim ** -0.5, *cols[3:],
                                conv.t().contiguous(), self._f32(get("A_log"), mix.heads), self._f32(get("dt_bias"), mix.heads),
                                self._f32(get("norm"), dv))
        o = get("o").reshape(self.width, mix.heads, mix.vdim)
        lw.out_cols = mix.heads * dv
        lw.w_o = self._weight(self._mat(o, (self.H, mix.heads, dv)).flatten(1), (self.H, lw.out_cols))

    def _pack_attention(self, lw, mix, get):
        # (in 16 bits heads as the tensor-core kernels take them; larger ones run the plain kernel)
        lw.pad = up(mix.dim, 64) if self.dtype == torch.bfloat16 and mix.dim <= 128 else up(mix.dim, 8)
        qk = torch.cat([get("q"), get("k")])
        lw.in_cols = up(qk.shape[0], 8)
        lw.w_in = self._weight(qk, (lw.in_cols, self.H))
        lw.bias = self._f32(torch.cat([get("q.b").reshape(-1), get("k.b").reshape(-1)]), lw.in_cols)
        i = np.arange(mix.rot // 2, dtype=np.float64)
        freq = mix.base ** (-2.0 * i / max(mix.rot, 1)) / mix.factor
        lw.inv_freq = torch.tensor(freq, dtype=torch.float32, device=self.device)
        lw.sink = self._f32(get("sink"), mix.heads)
        o = get("o").reshape(self.width, mix.heads, mix.dim)
        lw.out_cols = mix.heads * lw.pad
        lw.w_o = self._weight(self._mat(o, (self.H, mix.heads, lw.pad)).flatten(1), (self.H, lw.out_cols))

    # -- what the model is served with ----------------------------------------------------------------------------
    def new_cache(self, max_batch, max_total_seq_len, prefill_chunk, page_size=16, max_seq_len=None):
        attention, states = {}, {}
        for run, i in enumerate(self.config.runs):
            lw = self.layers[i]
            if isinstance(lw.mix, Attention):
                attention[run] = (lw.mix.kv_heads, lw.pad)
            else:
                r = lw.rule
                states[run] = {"S": ((r.heads, r.dim, r.vdim), torch.float32), "conv": ((r.taps, r.channels), self.dtype)}
        return HybridCache(attention, states, max_batch, max_total_seq_len, prefill_chunk, page_size, self.device,
                           max_seq_len=max_seq_len, dtype=self.dtype)

    def new_engine(self, kv, max_rows):
        return RelidraEngine(self, kv, max_rows)


class RelidraEngine(PlainEngine):
    def __init__(self, model: PackedRelidra, kv: HybridCache, max_rows: int):
        lws = model.layers
        shapes = [(model.H, model.V)]
        for lw in lws:
            shapes += [(model.H, lw.in_cols), (lw.out_cols, model.H)]
            shapes += [(model.H, lw.ffp), (lw.ffp, model.H)] if lw.ffp else []
        super().__init__(model, kv, max_rows, shapes)
        m, dev, T = model, model.device, self.max_rows
        act = dict(dtype=m.dtype, device=dev)
        self.emb = torch.zeros(T, m.H, dtype=torch.float32, device=dev)
        self.streams = torch.zeros(T, m.config.streams, m.H, dtype=torch.float32, device=dev)
        self.xn, self.y = torch.zeros(T, m.H, **act), torch.zeros(T, m.H, **act)
        widest = lambda f, cond=lambda lw: True: max([f(lw) for lw in lws if cond(lw)], default=8)
        delta, att = (lambda lw: isinstance(lw.mix, Delta)), (lambda lw: isinstance(lw.mix, Attention))
        self.proj = torch.zeros(T * widest(lambda lw: lw.in_cols), **act)
        self.mixed = torch.zeros(T * widest(lambda lw: lw.out_cols), **act)
        self.q = torch.zeros(T * widest(lambda lw: lw.out_cols, att), **act)
        self.act = torch.zeros(T * max(widest(lambda lw: lw.ffp), 8), **act)
        self._conv_cols, self._o_cols = widest(lambda lw: lw.rule.channels, delta), widest(lambda lw: lw.out_cols, delta)
        # prompt passes: segments of the recurrence, query tiles of <= 128 rows
        self.segs = torch.zeros(kv.max_batch, 4, dtype=torch.int32, device=dev)
        self.tiles = torch.zeros((T + 127) // 128 + kv.max_batch + 1, 4, dtype=torch.int32, device=dev)
        self._n_segs = self._n_tiles = self._max_seg = 0

    # -- prompt passes ------------------------------------------------------------------------------------------
    def _begin_prompt_pass(self, chunk):
        segs = [(self.kv.slot(sid), r0, n, p0) for sid, r0, n, p0 in chunk]
        tiles = [(s, r0 + off, min(128, n - off), p0 + off) for s, r0, n, p0 in segs for off in range(0, n, 128)]
        for dst, v in ((self.segs, segs), (self.tiles, tiles)):
            self._stage(dst.view(-1), np.asarray(v, dtype=np.int32).reshape(-1), torch.int32)
        self._n_segs, self._n_tiles, self._max_seg = len(segs), len(tiles), max(n for _, _, n, _ in segs)

    def _end_prompt_pass(self):
        self._n_segs = self._n_tiles = 0

    # -- pieces of a layer ----------------------------------------------------------------------------------------
    def _delta(self, T, lw, run, proj, out, decode):
        kv, r, eps = self.kv, lw.rule, self.m.config.eps
        S, ring, row_slot, row_pos = kv.state(run, "S"), kv.state(run, "conv"), self.row_slot[:T], self.row_pos[:T]
        if decode:
            return ops.delta_step(proj, r, eps, row_slot, row_pos, S, ring, out, status=self.status)
        xc = ops.short_conv(proj, r.conv, ring, row_slot, row_pos, self._grow("conv", self.max_rows * self._conv_cols)[:T * r.channels]
                            .view(T, r.channels))
        o = self._grow("o", self.max_rows * self._o_cols, torch.float32)[:T * lw.out_cols].view(T, lw.out_cols)
        if ops.delta_chunk_fits(r, self.m.dtype, self._max_seg):
            work = self._grow("chunks", ops.delta_chunk_workspace(T, self._n_segs, r.heads), torch.uint8)
            ops.delta_chunk(xc, proj, r, self.segs, self._n_segs, self._max_seg, S, ring, o, work, status=self.status)
        else:
            ops.delta_scan(xc, proj, r, self.segs, self._n_segs, S, ring, o)
        return ops.gated_rms(o, proj[:, r.g_col:], r.norm, r.heads, r.vdim_true, eps, out)

    def _attention(self, T, lw, run, proj, out, decode):
        kv, mix, eps = self.kv, lw.mix, self.m.config.eps
        row_slot, row_pos, K, V = self.row_slot[:T], self.row_pos[:T], kv.k_pages(run), kv.v_pages(run)
        if decode and ops.paged_attention_streams(self.m.dtype, lw.pad, kv.page_size):
            keys = min(self.max_keys, mix.chunk) if mix.chunk else self.max_keys
            splits = ops.paged_attention_splits(T, mix.heads, -(-keys // kv.page_size) + 1)
            nb = ops.paged_attention_workspace(T, mix.heads, lw.pad, splits) if splits > 1 else 0
            return ops.paged_attention_rms(proj, lw.bias, lw.inv_freq, mix.rot, mix.dim, eps, K, V, kv.block_table, row_slot, row_pos,
                                           mix.heads, mix.scale, out, chunk=mix.chunk, sink=lw.sink, n_splits=splits,
                                           work=self._grow("merge", nb, torch.uint8) if nb else None)
        q = ops.rotate_rms_append(proj, lw.bias, lw.inv_freq, mix.rot, mix.dim, eps, mix.scale,
                                  self.q[:T * lw.out_cols].view(T, lw.out_cols), K, V, kv.block_table, row_slot, row_pos, mix.heads,
                                  mix.kv_heads)
        if not decode and self.m.dtype == torch.bfloat16 and lw.pad in (64, 128):
            return ops.prefill_attention_masked(q, K, V, kv.block_table, self.tiles, self._n_tiles, mix.heads, 1.0, out,
                                                chunk=mix.chunk, sink=lw.sink, status=self.status)
        # (the scale is in the queries)
        return ops.paged_attention_masked(q, K, V, kv.block_table, row_slot, row_pos, mix.heads, 1.0, out, chunk=mix.chunk,
                                          sink=lw.sink)

    def _norm(self, T, w, read, src, add, rows=None):
        """Hands ``add`` = (rows, connection of the sublayer they come from) back to the streams and normalises the sum that
        ``read`` weighs into ``xn``; returns where the streams are."""
        m, c = self.m, self.m.config
        n = T if rows is None else rows.numel()
        y, back = add
        dst = self.streams[:T] if y is not None and rows is None else None
        ops.residual_streams_layernorm(y, src, read, w, c.eps, c.width, self.xn[:n], dst=dst, back=back, rows=rows)
        return src if dst is None else dst

    def forward(self, T, fused_append, use_lora=True, lm_rows=None, n_lm=None, hidden=None):
        """One pass over the T rows staged in ``tokens`` / ``row_slot`` / ``row_pos``; as :meth:`model.Engine.forward`.
        (``use_lora`` and the staged adapter slots mean nothing to a design without adapters.)"""
        m = self.m
        if not fused_append and not self._n_segs:
            raise RuntimeError("a prompt pass needs its segments: call _begin_prompt_pass first")
        if hidden is None:
            ops.embed(self.tokens[:T], m.embed, res=self.emb[:T])
        else:
            ops.embed(self.iota[:T], hidden, res=self.emb[:T])
        src, add, y = self.emb[:T], (None, None), self.y[:T]  # (until something comes back all streams are the embedding)
        for run, i in enumerate(m.config.runs):
            lw = m.layers[i]
            src = self._norm(T, lw.norm1, lw.hc1.read, src, add)
            proj = self._linear(self.xn[:T], lw.w_in, self.proj[:T * lw.in_cols].view(T, lw.in_cols))
            mixer = self._delta if isinstance(lw.mix, Delta) else self._attention
            out = mixer(T, lw, run, proj, self.mixed[:T * lw.out_cols].view(T, lw.out_cols), fused_append)
            add = (self._linear(out, lw.w_o, y), lw.hc1.back)
            if lw.ffp:
                src = self._norm(T, lw.norm2, lw.hc2.read, src, add)
                a = self._linear(self.xn[:T], lw.up, self.act[:T * lw.ffp].view(T, lw.ffp), ACT_GELU)
                add = (self._linear(a, lw.down, y), lw.hc2.back)
        rows = None if lm_rows is None else lm_rows[:n_lm]
        n = T if rows is None else n_lm
        self._norm(T, m.norm, m.sum_streams, src, add, rows)
        self._linear(self.xn[:n], m.head, self.logits[:n], OUT_F32)
        ops.argmax(self.logits[:n], out=self.next_tok[:n])
        return self.logits[:n], self.next_tok[:n]
