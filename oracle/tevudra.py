"""Plain Tevudra decoder in PyTorch on the CPU: one function per mechanism, no cache, no batching.

The checker of the CUDA path.  It shares no code with the package: every function below restates its equation on
whole sequences in the dtype of its inputs (float64 or float32).  ``params`` is a dict of tensors under the names of
the checkpoint format.
"""
from __future__ import annotations

import math

import torch


def dyt(x, alpha, w, b):
    """Dynamic tanh: y = w * tanh(alpha x) + b, elementwise."""
    return w * torch.tanh(alpha * x) + b


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def relu2(z):
    return torch.clamp(z, min=0) ** 2


def gelu_erf(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


def feed_forward(h, up, down, act):
    return act(h @ up.T) @ down.T


def route(h, w, b, top):
    """(indices [n, top], weights [n, top]): the ``top`` largest logits and the softmax over exactly those."""
    z = h @ w.T + b
    val, idx = torch.topk(z, top, dim=-1)
    return idx, torch.softmax(val, -1)


def moe(h, router_w, router_b, top, experts, shared=None):
    """experts: list of (up, down); shared: (up, down) or None."""
    idx, wt = route(h, router_w, router_b, top)
    out = torch.zeros_like(h)
    for n in range(h.shape[0]):
        for k in range(top):
            up, down = experts[int(idx[n, k])]
            out[n] += wt[n, k] * feed_forward(h[n:n + 1], up, down, gelu_erf)[0]
    if shared is not None:
        out = out + feed_forward(h, shared[0], shared[1], gelu_erf)
    return out


def latent(h, w_dkv, w_norm, eps):
    return rms(h @ w_dkv.T, w_norm, eps)


def latent_attention(h, c, w_q, w_uk, w_uv, w_g, w_o, heads, dim, vdim, scale):
    """h [n, width] inputs, c [n, rank] latents of the same positions (this layer's own or another layer's)."""
    n = h.shape[0]
    q = (h @ w_q.T).view(n, heads, dim)
    k = (c @ w_uk.T).view(n, heads, dim)
    v = (c @ w_uv.T).view(n, heads, vdim)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    seen = torch.ones(n, n, dtype=torch.bool).tril()
    p = torch.softmax(s.masked_fill(~seen, float("-inf")), -1)
    o = torch.einsum("hij,jhd->ihd", p, v) * torch.sigmoid(h @ w_g.T)[:, :, None]
    return o.reshape(n, heads * vdim) @ w_o.T


class OracleTevudra:
    """``margin`` (after a forward): per token the smallest distance, over the layers, between the last chosen expert's
    logit and the first one left out -- a 16-bit path may choose the other one where it is small."""

    def __init__(self, config, params, dtype=torch.float64):
        self.cfg = config
        self.p = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in params.items()}

    def _norm(self, name, x):
        p = self.p
        return dyt(x, p[name + ".alpha"], p[name], p[name + ".b"])

    def _mlp(self, pre, m, h):
        p = self.p
        if m["kind"] == "moe" and m["router"]["top"] < m["router"]["experts"]:
            z = torch.sort(h @ p[pre + "router"].T + p[pre + "router.b"], dim=-1, descending=True).values
            top = m["router"]["top"]
            self.margin = torch.minimum(self.margin, z[:, top - 1] - z[:, top])
        if m["kind"] == "dense":
            return feed_forward(h, p[pre + "up"], p[pre + "down"], relu2)
        n_exp = m["router"]["experts"]
        ex = [(p[f"{pre}e{e}.up"], p[f"{pre}e{e}.down"]) for e in range(n_exp)]
        sh = (p[pre + "shared.up"], p[pre + "shared.down"]) if m.get("shared") else None
        return moe(h, p[pre + "router"], p[pre + "router.b"], m["router"]["top"], ex, sh)

    def forward(self, tokens):
        """(logits [n, vocab], residual stream after every layer [layers, n, width])."""
        p, eps = self.p, self.cfg["norm"]["eps"]
        x = p["embed"][torch.as_tensor(tokens, dtype=torch.long)]
        lat, stream = {}, []
        self.margin = torch.full((len(tokens),), float("inf"), dtype=x.dtype)
        for i, layer in enumerate(self.cfg["layers"]):
            m, pre = layer["mixer"], f"l{i}."
            h = self._norm(pre + "norm1", x)
            src = m.get("kv_from", i)
            if src == i:
                lat[i] = latent(h, p[pre + "mix.dkv"], p[pre + "mix.dkv.norm"], eps)
            x = x + latent_attention(h, lat[src], p[pre + "mix.q"], p[pre + "mix.uk"], p[pre + "mix.uv"],
                                     p[pre + "mix.g"], p[pre + "mix.o"], m["heads"], m["dim"], m["vdim"], m["scale"])
            if layer.get("mlp"):
                x = x + self._mlp(pre + "mlp.", layer["mlp"], self._norm(pre + "norm2", x))
            stream.append(x)
        logits = self._norm("final.norm", x) @ p["head"].T
        return logits, torch.stack(stream)

    def greedy(self, prompt, n):
        """``n`` greedily chosen tokens after ``prompt``, and the logits each was chosen from."""
        toks, lgs = list(prompt), []
        for _ in range(n):
            lg = self.forward(toks)[0][-1]
            lgs.append(lg)
            toks.append(int(lg.argmax()))
        return toks[len(prompt):], torch.stack(lgs)
