"""Small Tevudra configurations with random weights for the tests."""
import math

import torch


def layer(heads, dim, vdim, rank, scale=None, kv_from=None, mlp=None):
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": dim ** -0.5 if scale is None else scale}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Tevudra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    # nothing a multiple of anything, every layer its own sizes, one layer without feed-forward, latents read two layers on
    "odd": config(84, 101, [
        layer(3, 20, 28, 44, mlp=moe(36, 7, 3, 52)),
        layer(5, 12, 9, 30, scale=0.4, mlp=None),
        layer(2, 33, 17, 44, kv_from=0, mlp=dense(150)),
        layer(4, 24, 40, 30, kv_from=1, scale=0.17, mlp=moe(20, 5, 1)),
    ]),
    # heads beyond one group of 32, a rank of several chunks, every expert chosen, eps that matters
    "wide": config(160, 260, [
        layer(36, 16, 8, 264, mlp=dense(96)),
        layer(17, 64, 128, 264, kv_from=0, mlp=moe(64, 4, 4, 32)),
    ], eps=0.05),
    # one head, one expert, head sizes beyond the tensor-core prompt attention, a rank beyond the tensor-core decode kernel
    "single": config(72, 64, [
        layer(1, 144, 136, 520, mlp=moe(40, 1, 1, 24)),
        layer(1, 8, 8, 8, mlp=dense(8)),
    ]),
    # several layers on one latent
    "shared": config(128, 300, [
        layer(4, 48, 48, 128, mlp=dense(200)),
        layer(4, 48, 48, 128, kv_from=0, mlp=moe(48, 12, 4, 48)),
        layer(8, 24, 32, 128, kv_from=0, mlp=moe(24, 9, 2)),
    ]),
}


def weights(cfg, seed=0, sharp=3.0):
    """Random bf16 tensors under the checkpoint's names.  ``sharp`` scales the queries: scores then differ by several
    units, so that a single key decides a head's result and a wrong or missing one shows."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s, k=1.0: (torch.randn(*s, generator=g) * k).bfloat16()
    mat = lambda o, i, k=1.0: rnd(o, i, k=k / math.sqrt(i))
    W, V = cfg["width"], cfg["vocab"]
    p = {"embed": rnd(V, W), "head": mat(V, W)}

    def norm(name):
        p[name], p[name + ".b"] = (1 + 0.2 * torch.randn(W, generator=g)).bfloat16(), rnd(W, k=0.2)
        p[name + ".alpha"] = torch.tensor(float(0.4 + 0.3 * torch.rand((), generator=g))).bfloat16()

    norm("final.norm")
    for i, layer_ in enumerate(cfg["layers"]):
        m, pre = layer_["mixer"], f"l{i}."
        norm(pre + "norm1")
        H, R = m["heads"], m["kv_rank"]
        p[pre + "mix.q"] = mat(H * m["dim"], W, sharp / (m["scale"] * math.sqrt(m["dim"])))
        if "kv_from" not in m:
            p[pre + "mix.dkv"], p[pre + "mix.dkv.norm"] = mat(R, W), (1 + 0.3 * torch.randn(R, generator=g)).bfloat16()
        p[pre + "mix.uk"], p[pre + "mix.uv"] = mat(H * m["dim"], R), mat(H * m["vdim"], R)
        p[pre + "mix.g"], p[pre + "mix.o"] = mat(H, W), mat(W, H * m["vdim"], 6.0)
        f = layer_.get("mlp")
        if not f:
            continue
        norm(pre + "norm2")
        ff = lambda name, n: p.update({name + ".up": mat(n, W), name + ".down": mat(W, n)})
        if f["kind"] == "dense":
            ff(pre + "mlp", f["ff"])
            continue
        E = f["router"]["experts"]
        p[pre + "mlp.router"], p[pre + "mlp.router.b"] = mat(E, W, 5.0), rnd(E, k=0.5)
        for e in range(E):
            ff(f"{pre}mlp.e{e}", f["expert"]["ff"])
        if f.get("shared"):
            ff(pre + "mlp.shared", f["shared"]["ff"])
    return p


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


def check(got, want, dtype, margin=None):
    """Every row agrees; in 16 bits rows whose choice of experts is a close call are left out (they must be few)."""
    err = error(got, want)
    if dtype == torch.float32:
        assert float(err.max()) < 2e-4, err
        return
    if margin is not None:
        sure = margin > 0.25
        assert len(err) < 8 or int(sure.sum()) > len(err) // 2
        err = err[sure]
    assert len(err) == 0 or float(err.max()) < 0.06, err


def error(got, want):
    """Per row: root mean square of the difference (mean taken off) over that of the expected logits."""
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()
