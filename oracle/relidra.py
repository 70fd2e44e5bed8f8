"""Plain Relidra decoder in PyTorch on the CPU: one function per mechanism, no cache, no batching.

What the CUDA path is compared with.  It shares no code with the package: every function below restates its equation on
whole sequences in the dtype of its inputs (float64 or float32).  ``params`` is a dict of tensors under the names of
the checkpoint format.
"""
from __future__ import annotations

import math

import torch


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1 + torch.exp(-z))


def gelu_erf(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


def feed_forward(h, up, down):
    return gelu_erf(h @ up.T) @ down.T


def hyper_connect(streams, w_in, w_mix, w_out, sublayer):
    """streams [s, n, width]; ``sublayer`` maps the weighted sum of the streams to what is handed back to all of them."""
    u = sum(w_in[s] * streams[s] for s in range(len(streams)))
    y = sublayer(u)
    return torch.stack([sum(w_mix[s, t] * streams[s] for s in range(len(streams))) + w_out[t] * y for t in range(len(streams))])


def short_conv(x, taps):
    """x [n, channels], taps [channels, K]: a channel's own row weighs its last K inputs, taps[:, K - 1] the newest."""
    n, K = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for i in range(n):
        for k in range(K):
            j = i - (K - 1) + k
            if j >= 0:
                out[i] += taps[:, k] * x[j]
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_decay(a, A_log, dt_bias):
    z = a + dt_bias
    return torch.exp(-torch.exp(A_log) * torch.log1p(torch.exp(-z.abs())) - torch.exp(A_log) * torch.clamp(z, min=0))


def delta_rule(q, k, v, g, beta, state=None):
    """One head.  q, k [n, dim], v [n, vdim], g, beta [n] -> outputs [n, vdim], state [dim, vdim]."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(q.shape[0]):
        S = g[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + k[t][:, None] * u[None, :]
        out.append(S.T @ q[t])
    return torch.stack(out), S


def delta_mixer(h, p, pre, heads, kv_heads, dim, vdim, eps):
    n = h.shape[0]
    conv = lambda name: silu(short_conv(h @ p[pre + name].T, p[pre + name + ".conv"]))
    q, k = unit(conv("q").view(n, kv_heads, dim)) * dim ** -0.5, unit(conv("k").view(n, kv_heads, dim))
    v = conv("v").view(n, heads, vdim)
    beta = 1 / (1 + torch.exp(-(h @ p[pre + "b"].T)))
    g = delta_decay(h @ p[pre + "a"].T, p[pre + "A_log"], p[pre + "dt_bias"])
    gate = silu(h @ p[pre + "g"].T).view(n, heads, vdim)
    o = torch.zeros(n, heads, vdim, dtype=h.dtype)
    for x in range(heads):
        y = x // (heads // kv_heads)
        o[:, x] = delta_rule(q[:, y], k[:, y], v[:, x], g[:, x], beta[:, x])[0]
    return (rms(o, eps) * p[pre + "norm"] * gate).reshape(n, heads * vdim) @ p[pre + "o"].T


def rotate(x, pos, dims, base, factor):
    """x [n, heads, dim]: values i and i + dims / 2 of a head turn together, for i below dims / 2."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) / factor for i in range(half)], dtype=x.dtype)
    a = (pos.to(x.dtype)[:, None] * f)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), x[..., dims:]], -1)


def chunk_mask(n, size):
    i = torch.arange(n)
    seen = i[None, :] <= i[:, None]
    return seen if size is None else seen & (i[None, :] // size == i[:, None] // size)


def sink_softmax(s, sink):
    """s [heads, n, n] (-inf where not seen), sink [heads]: a key without a value that every query sees."""
    full = torch.cat([s, sink[:, None, None].expand(-1, s.shape[1], 1)], -1)
    return torch.softmax(full, -1)[..., :-1]


def attention_mixer(h, p, pre, heads, kv_heads, dim, rot, scale, chunk, eps):
    n, rep = h.shape[0], heads // kv_heads
    q = (h @ p[pre + "q"].T + p[pre + "q.b"]).view(n, heads, dim)
    k = (h @ p[pre + "k"].T + p[pre + "k.b"]).view(n, kv_heads, dim)
    v = k
    pos = torch.arange(n)
    q, k = (rms(rotate(x, pos, *rot), eps) for x in (q, k))
    k, v = k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    w = sink_softmax(s.masked_fill(~chunk_mask(n, chunk), float("-inf")), p[pre + "sink"])
    return torch.einsum("hij,jhd->ihd", w, v).reshape(n, heads * dim) @ p[pre + "o"].T


class OracleRelidra:
    def __init__(self, config, params, dtype=torch.float64):
        self.cfg = config
        self.p = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in params.items()}

    def order(self):
        """Layer indices in the order they run."""
        n, loop = len(self.cfg["layers"]), self.cfg.get("loop")
        if not loop:
            return list(range(n))
        a, b = loop["start"], loop["stop"]
        return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))

    def _mixer(self, i, h):
        layer, p, eps, pre = self.cfg["layers"][i], self.p, self.cfg["norm"]["eps"], f"l{i}.mix."
        m = layer["mixer"]
        if layer["type"] == "delta":
            return delta_mixer(h, p, pre, m["heads"], m["kv_heads"], m["dim"], m["vdim"], eps)
        r = m["rot"]
        factor = r["scaling"]["factor"] if r.get("scaling") else 1.0
        return attention_mixer(h, p, pre, m["heads"], m["kv_heads"], m["dim"], (r["dims"], r["base"], factor), m["scale"],
                               m["mask"]["size"] if m.get("mask") else None, eps)

    def forward(self, tokens):
        """(logits [n, vocab], sum of the streams after every layer run [runs, n, width])."""
        p, eps = self.p, self.cfg["norm"]["eps"]
        x = p["embed"][torch.as_tensor(tokens, dtype=torch.long)]
        x = x.expand(self.cfg["streams"], -1, -1)
        stream = []
        for i in self.order():
            pre = f"l{i}."
            hc = lambda q: (p[f"{pre}hc{q}.in"], p[f"{pre}hc{q}.mix"], p[f"{pre}hc{q}.out"])
            x = hyper_connect(x, *hc(1), lambda u: self._mixer(i, layer_norm(u, p[pre + "norm1"], eps)))
            if self.cfg["layers"][i].get("mlp"):
                x = hyper_connect(x, *hc(2), lambda u: feed_forward(layer_norm(u, p[pre + "norm2"], eps),
                                                                    p[pre + "mlp.up"], p[pre + "mlp.down"]))
            stream.append(x.sum(0))
        logits = layer_norm(x.sum(0), p["final.norm"], eps) @ p["embed"].T
        return logits, torch.stack(stream)

    def greedy(self, prompt, n):
        """``n`` greedily chosen tokens after ``prompt``, and the logits each was chosen from."""
        toks, lgs = list(prompt), []
        for _ in range(n):
            lg = self.forward(toks)[0][-1]
            lgs.append(lg)
            toks.append(int(lg.argmax()))
        return toks[len(prompt):], torch.stack(lgs)
