"""Small Relidra configurations with random weights for the tests."""
import math

import torch

from tevudra_cases import error, tokens  # noqa: F401  (same meaning here)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def delta(heads, kv_heads, dim, vdim, taps, ff=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps},
            "mlp": dense(ff) if ff else None}


def attention(heads, kv_heads, dim, rot, chunk, base=10000.0, factor=1.0, scale=None, ff=None):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": chunk},
                      "rot": {"base": base, "dims": rot, "scaling": {"factor": factor}},
                      "scale": 2 / math.sqrt(dim) if scale is None else scale},
            "mlp": dense(ff) if ff else None}


def config(width, vocab, streams, layers, loop=None, eps=1e-5):
    c = {"architecture": "Relidra", "width": width, "vocab": vocab, "streams": streams, "norm": {"eps": eps}, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CONFIGS = {
    # nothing a multiple of anything, every layer its own sizes, a loop in the middle
    "odd": config(84, 101, 3, [
        delta(6, 2, 20, 12, 3, ff=150),
        attention(4, 2, 36, 20, 23, base=700.0, factor=2.5, scale=0.4),
        delta(3, 3, 33, 41, 5),
        attention(5, 1, 72, 72, 40, factor=8.0, ff=36),
    ], loop=(1, 3, 2)),
    # one stream, wide heads, a chunk of one tile, eps that matters, attention first
    "wide": config(160, 260, 1, [
        attention(8, 8, 128, 64, 128, ff=96),
        delta(16, 4, 128, 136, 4, ff=64),
    ], eps=0.05),
    # single heads, one tap, heads beyond the tensor-core attention, chunks shorter than a page, a loop of one pass
    "single": config(72, 64, 4, [
        delta(1, 1, 8, 8, 1),
        attention(1, 1, 144, 100, 7, base=50.0, scale=-0.2, ff=8),
        delta(2, 1, 200, 8, 2, ff=24),
    ], loop=(0, 1, 1)),
    # everything in the loop
    "deep": config(128, 300, 2, [
        delta(4, 2, 40, 64, 4),
        attention(4, 2, 64, 32, 48, base=2000.0, factor=4.0, ff=200),
    ], loop=(0, 2, 3)),
    # more streams than the unrolled kernels have
    "streams": config(64, 90, 6, [
        attention(2, 1, 16, 16, 30, ff=40),
        delta(2, 2, 16, 24, 4),
        attention(2, 2, 24, 8, 17),
    ]),
}


def weights(cfg, seed=7):
    """Random bf16 tensors under the checkpoint's names.  Scores differ by several units, sinks are as large as a whole
    chunk's sum, most decays are close to one and the convolutions' older taps weigh as much as the current one: a single
    wrong key, a lost sink, a lost state or a lost convolution input changes the logits."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s, k=1.0: (torch.randn(*s, generator=g) * k).bfloat16()
    uni = lambda n, a, b: (a + (b - a) * torch.rand(n, generator=g)).bfloat16()
    mat = lambda o, i, k=1.0: rnd(o, i, k=k / math.sqrt(i))
    W, n = cfg["width"], cfg["streams"]
    p = {"embed": rnd(cfg["vocab"], W)}
    norm = lambda name: p.update({name: (1 + 0.2 * torch.randn(W, generator=g)).bfloat16()})

    def connection(name):
        p[name + ".in"], p[name + ".out"] = uni(n, 0.3, 1.0), uni(n, 0.3, 0.8)
        p[name + ".mix"] = (0.8 * torch.eye(n) + 0.9 * torch.randn(n, n, generator=g) / n).bfloat16()

    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        m, pre = layer["mixer"], f"l{i}."
        H, G, d, x = m["heads"], m["kv_heads"], m["dim"], pre + "mix."
        norm(pre + "norm1")
        connection(pre + "hc1")
        if layer["type"] == "delta":
            v = m["vdim"]
            for name, rows in (("q", G * d), ("k", G * d), ("v", H * v)):
                p[x + name], p[x + name + ".conv"] = mat(rows, W), (0.2 + 0.6 * torch.randn(rows, m["conv"], generator=g)).bfloat16()
            p[x + "g"], p[x + "b"], p[x + "a"] = mat(H * v, W), mat(H, W), mat(H, W)
            p[x + "A_log"], p[x + "dt_bias"] = uni(H, -4.0, 0.5), uni(H, -3.0, -1.0)
            p[x + "norm"], p[x + "o"] = (1 + 0.2 * torch.randn(v, generator=g)).bfloat16(), mat(W, H * v, 1.2)
        else:
            for name, rows in (("q", H * d), ("k", G * d)):
                p[x + name], p[x + name + ".b"] = mat(rows, W), rnd(rows, k=0.4)
            p[x + "sink"], p[x + "o"] = (4 + torch.randn(H, generator=g)).bfloat16(), mat(W, H * d, 2.0)
        if layer.get("mlp"):
            norm(pre + "norm2")
            connection(pre + "hc2")
            ff = layer["mlp"]["ff"]
            p[pre + "mlp.up"], p[pre + "mlp.down"] = mat(ff, W), mat(W, ff)
    return p


def check(got, want, dtype):
    err = error(got, want)
    assert float(err.max()) < (2e-4 if dtype == torch.float32 else 0.06), err
