"""Seeded synthetic models, adapters and request batches.

The reference runs pretrained Llama weights, adapter files written by
``init_peft_weights/lora_weights.py`` and one English prompt replicated over
the batch (``huggingface/generation/gen_lora.py:96-98``); none of those are
available offline, so every workload here is random data with the same
shapes, drawn from fixed seeds: tokens 0, base weights 1, adapters 2,
adapter ids 3, prompt lengths 4.
"""
from __future__ import annotations

import math

import numpy as np
import torch

SEED_TOKENS, SEED_WEIGHTS, SEED_ADAPTERS, SEED_IDS, SEED_LENS = 0, 1, 2, 3, 4

ATTN_PROJ = ("q_proj", "k_proj", "v_proj", "o_proj")
MLP_PROJ = ("gate_proj", "up_proj", "down_proj")


def llama_config(name: str) -> dict:
    """Field names of ``tvm/llama_auto_batcher/llama_for_causal_lm.py:10-21``."""
    base = dict(rms_norm_eps=1e-5, vocab_size=32000, rope_theta=10000.0)
    if name == "tiny":  # the CPU-runnable plumbing case
        return dict(base, name=name, hidden_size=256, intermediate_size=688, num_attention_heads=4,
                    num_hidden_layers=2, num_key_value_heads=4, head_dim=64)
    if name == "llama2-7b":
        return dict(base, name=name, hidden_size=4096, intermediate_size=11008, num_attention_heads=32,
                    num_hidden_layers=32, num_key_value_heads=32, head_dim=128)
    if name == "llama2-13b":
        return dict(base, name=name, hidden_size=5120, intermediate_size=13824, num_attention_heads=40,
                    num_hidden_layers=40, num_key_value_heads=40, head_dim=128)
    raise KeyError(name)


def proj_shape(cfg: dict, proj: str):
    """(out_features, in_features) of a projection."""
    H, I = cfg["hidden_size"], cfg["intermediate_size"]
    D, Hq, Hkv = cfg["head_dim"], cfg["num_attention_heads"], cfg["num_key_value_heads"]
    return {
        "q_proj": (Hq * D, H), "k_proj": (Hkv * D, H), "v_proj": (Hkv * D, H), "o_proj": (H, Hq * D),
        "gate_proj": (I, H), "up_proj": (I, H), "down_proj": (H, I),
    }[proj]


def _gen(seed, device):
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    return g


def base_weights(cfg: dict, dtype=torch.float32, device="cpu", n_layers=None) -> dict:
    """HF-named state dict, every matrix ~ N(0, 0.02), norm weights 1 + N(0, 0.02)."""
    g = _gen(SEED_WEIGHTS, device)
    H, V = cfg["hidden_size"], cfg["vocab_size"]
    L = cfg["num_hidden_layers"] if n_layers is None else n_layers

    def mat(o, i):
        return (torch.randn(o, i, generator=g, device=device, dtype=torch.float32) * 0.02).to(dtype)

    def vec(n):
        return (1.0 + 0.02 * torch.randn(n, generator=g, device=device, dtype=torch.float32)).to(dtype)

    w = {"model.embed_tokens.weight": mat(V, H)}
    for l in range(L):
        p = f"model.layers.{l}."
        for proj in ATTN_PROJ:
            w[p + f"self_attn.{proj}.weight"] = mat(*proj_shape(cfg, proj))
        for proj in MLP_PROJ:
            w[p + f"mlp.{proj}.weight"] = mat(*proj_shape(cfg, proj))
        w[p + "input_layernorm.weight"] = vec(H)
        w[p + "post_attention_layernorm.weight"] = vec(H)
    w["model.norm.weight"] = vec(H)
    w["lm_head.weight"] = mat(V, H)
    return w


def lora_adapters(cfg: dict, n_adapters: int, ranks, targets=ATTN_PROJ, dtype=torch.float32,
                  device="cpu", n_layers=None):
    """Adapter dicts keyed like the reference's adapter files
    (``init_peft_weights/lora_weights.py:18-23``): ``lora_A`` [r,in] ~ kaiming
    uniform(a=sqrt 5) = U(+-1/sqrt(in)), ``lora_B`` [out,r] ~ N(0, 0.02).
    ``ranks`` is an int or a sequence cycled over the adapters."""
    g = _gen(SEED_ADAPTERS, device)
    L = cfg["num_hidden_layers"] if n_layers is None else n_layers
    ranks = [ranks] if isinstance(ranks, int) else list(ranks)
    out = []
    for a in range(n_adapters):
        r = ranks[a % len(ranks)]
        d = {}
        for l in range(L):
            for proj in targets:
                blk = "self_attn" if proj in ATTN_PROJ else "mlp"
                o, i = proj_shape(cfg, proj)
                bound = 1.0 / math.sqrt(i)
                A = (torch.rand(r, i, generator=g, device=device, dtype=torch.float32) * 2 - 1) * bound
                B = torch.randn(o, r, generator=g, device=device, dtype=torch.float32) * 0.02
                d[f"layers.{l}.{blk}.{proj}.lora_A.weight"] = A.to(dtype)
                d[f"layers.{l}.{blk}.{proj}.lora_B.weight"] = B.to(dtype)
        out.append(d)
    return out


def tevudra_config(name: str) -> dict:
    """Tevudra shapes with layers like a real model's: four layers, two latents, dense and mixture-of-experts in turn."""
    w, heads, ff, experts, eff, top, shared = {"tevudra-2048": (2048, 16, 8192, 64, 1408, 6, 2816),
                                               "tevudra-4096": (4096, 32, 16384, 32, 2048, 4, 4096)}[name]
    def layer(i):
        mixer = {"heads": heads, "dim": 128, "vdim": 128, "kv_rank": 512, "scale": 128 ** -0.5}
        if i % 2:
            mixer["kv_from"] = i - 1
            mlp = {"kind": "moe", "expert": {"ff": eff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}
        else:
            mlp = {"kind": "dense", "ff": ff}
        return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}
    return {"architecture": "Tevudra", "name": name, "vocab": 32000, "width": w, "norm": {"eps": 1e-6},
            "layers": [layer(i) for i in range(4)]}


def tevudra_weights(cfg: dict, dtype=torch.bfloat16, device="cpu") -> dict:
    """Random weights of a Tevudra configuration: matrices ~ N(0, 1/in), norm weights 1 + N(0, 0.02), alpha 0.5."""
    g = _gen(SEED_WEIGHTS, device)
    rnd = lambda *s: torch.randn(*s, generator=g, device=device, dtype=torch.float32)
    mat = lambda o, i: (rnd(o, i) / math.sqrt(i)).to(dtype)
    W, V = cfg["width"], cfg["vocab"]
    p = {"embed": rnd(V, W).to(dtype), "head": mat(V, W)}

    def norm(name):
        p[name], p[name + ".b"] = (1 + 0.02 * rnd(W)).to(dtype), (0.02 * rnd(W)).to(dtype)
        p[name + ".alpha"] = torch.tensor(0.5, device=device).to(dtype)

    def feed_forward(name, ff):
        p[name + ".up"], p[name + ".down"] = mat(ff, W), mat(W, ff)

    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        m, f, mix = layer["mixer"], layer["mlp"], f"l{i}.mix."
        H, R = m["heads"], m["kv_rank"]
        norm(f"l{i}.norm1")
        p[mix + "q"], p[mix + "g"], p[mix + "o"] = mat(H * m["dim"], W), mat(H, W), mat(W, H * m["vdim"])
        p[mix + "uk"], p[mix + "uv"] = mat(H * m["dim"], R), mat(H * m["vdim"], R)
        if "kv_from" not in m:
            p[mix + "dkv"], p[mix + "dkv.norm"] = mat(R, W), (1 + 0.02 * rnd(R)).to(dtype)
        if f is None:
            continue
        norm(f"l{i}.norm2")
        if f["kind"] == "dense":
            feed_forward(f"l{i}.mlp", f["ff"])
            continue
        p[f"l{i}.mlp.router"], p[f"l{i}.mlp.router.b"] = (4 * mat(f["router"]["experts"], W)).to(dtype), (0.1 * rnd(f["router"]["experts"])).to(dtype)
        for e in range(f["router"]["experts"]):
            feed_forward(f"l{i}.mlp.e{e}", f["expert"]["ff"])
        if f.get("shared"):
            feed_forward(f"l{i}.mlp.shared", f["shared"]["ff"])
    return p


def relidra_config(name: str) -> dict:
    """Relidra shapes with layers like a real model's: delta-rule and attention layers in turn, four query heads to a key head."""
    w, heads, ff, streams = {"relidra-2048": (2048, 16, 8192, 2), "relidra-4096": (4096, 32, 16384, 4)}[name]
    delta = {"type": "delta", "mixer": {"heads": heads, "kv_heads": heads // 2, "dim": 128, "vdim": 128, "conv": 4}}
    att = {"type": "attention", "mixer": {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                          "mask": {"size": 16384}, "rot": {"base": 500000.0, "dims": 128, "scaling": {"factor": 1.0}}}}
    return {"architecture": "Relidra", "name": name, "vocab": 32000, "width": w, "streams": streams, "norm": {"eps": 1e-6},
            "layers": [dict((att if i % 2 else delta), mlp={"kind": "dense", "ff": ff}) for i in range(4)]}


def relidra_weights(cfg: dict, dtype=torch.bfloat16, device="cpu") -> dict:
    """Random weights of a Relidra configuration: matrices ~ N(0, 1/in), norm weights 1 + N(0, 0.02), streams that mostly stay
    themselves."""
    g = _gen(SEED_WEIGHTS, device)
    rnd = lambda *s: torch.randn(*s, generator=g, device=device, dtype=torch.float32)
    mat = lambda o, i: (rnd(o, i) / math.sqrt(i)).to(dtype)
    W, n = cfg["width"], cfg["streams"]
    p = {"embed": rnd(cfg["vocab"], W).to(dtype), "final.norm": (1 + 0.02 * rnd(W)).to(dtype)}

    def sublayer(i, q):
        p[f"l{i}.norm{q}"] = (1 + 0.02 * rnd(W)).to(dtype)
        hc = f"l{i}.hc{q}."
        p[hc + "in"], p[hc + "out"] = (1 / n + 0.1 * rnd(n)).to(dtype), (0.5 + 0.1 * rnd(n)).to(dtype)
        p[hc + "mix"] = (torch.eye(n, device=device) + 0.1 * rnd(n, n)).to(dtype)

    for i, layer in enumerate(cfg["layers"]):
        m, x = layer["mixer"], f"l{i}.mix."
        H, G, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        sublayer(i, 1)
        for name, rows in (("q", G * d), ("k", G * d), ("v", H * v)) if layer["type"] == "delta" else (("q", H * d), ("k", G * d)):
            p[x + name] = mat(rows, W)
            if layer["type"] == "delta":
                p[x + name + ".conv"] = (rnd(rows, m["conv"]) / math.sqrt(m["conv"])).to(dtype)
            else:
                p[x + name + ".b"] = (0.1 * rnd(rows)).to(dtype)
        p[x + "o"] = mat(W, H * v)
        if layer["type"] == "delta":
            p[x + "g"], p[x + "b"], p[x + "a"] = mat(H * v, W), mat(H, W), mat(H, W)
            p[x + "A_log"], p[x + "dt_bias"], p[x + "norm"] = rnd(H).to(dtype) - 2, rnd(H).to(dtype) - 2, (1 + 0.02 * rnd(v)).to(dtype)
        else:
            p[x + "sink"] = rnd(H).to(dtype)
        if layer["mlp"]:
            sublayer(i, 2)
            p[f"l{i}.mlp.up"], p[f"l{i}.mlp.down"] = mat(layer["mlp"]["ff"], W), mat(W, layer["mlp"]["ff"])
    return p


def adapter_ids_uniform(n_requests: int, n_adapters: int) -> np.ndarray:
    return np.random.default_rng(SEED_IDS).integers(0, n_adapters, n_requests).astype(np.int32)


def adapter_ids_zipf(n_requests: int, n_adapters: int, s: float = 1.1) -> np.ndarray:
    p = np.arange(1, n_adapters + 1, dtype=np.float64) ** (-s)
    p /= p.sum()
    return np.random.default_rng(SEED_IDS).choice(n_adapters, size=n_requests, p=p).astype(np.int32)


def request_mix(request_type: str, batch_size: int, seed: int = SEED_IDS) -> np.ndarray:
    """The reference's three request mixes (``huggingface/generation/gen_lora.py:77-85``): ``uniform`` = sorted
    draws from ``[0, ceil(sqrt(B)))`` (same-adapter rows contiguous), ``distinct`` = every request its own adapter,
    ``identical`` = one adapter for all.  Seeded (the reference draws from numpy's global generator)."""
    if request_type == "uniform":
        hi = int(np.ceil(np.sqrt(batch_size)))
        return np.sort(np.random.default_rng(seed).integers(0, hi, batch_size)).astype(np.int32)
    if request_type == "distinct":
        return np.arange(batch_size, dtype=np.int32)
    if request_type == "identical":
        return np.zeros(batch_size, dtype=np.int32)
    raise ValueError(f"unknown request_type {request_type}")


def request_mix_by_rank(request_type: str, batch_size: int, num_seqs_per_adapter, lora_ranks, seed: int = SEED_IDS):
    """The auto-batcher driver's batch (``tvm/llama_auto_batcher/main.py:24-35``): one group of requests per adapter
    rank, weight ids inside a group drawn per ``request_type``, and ``batch_size - sum(groups)`` requests WITHOUT
    adapter padded in front.  Returns ``(ranks, wids)``, each ``[batch_size]`` with -1 for the padding rows."""
    if sum(num_seqs_per_adapter) > batch_size:
        raise ValueError("more adapter requests than the batch holds")
    ranks = [r for n, r in zip(num_seqs_per_adapter, lora_ranks) for _ in range(n)]
    if request_type == "identical":
        wids = [0] * sum(num_seqs_per_adapter)
    else:
        wids = [int(w) for g, n in enumerate(num_seqs_per_adapter) for w in request_mix(request_type, n, seed + g)]
    pad = [-1] * (batch_size - sum(num_seqs_per_adapter))
    return np.asarray(pad + ranks, dtype=np.int32), np.asarray(pad + wids, dtype=np.int32)


def prompts(n_requests: int, length: int, vocab: int) -> np.ndarray:
    return np.random.default_rng(SEED_TOKENS).integers(0, vocab, (n_requests, length)).astype(np.int32)


def prompt_lengths(n_requests: int, lo: int, hi: int) -> np.ndarray:
    return np.random.default_rng(SEED_LENS).integers(lo, hi + 1, n_requests).astype(np.int32)


def operator_case(T: int, in_features=4096, out_features=4096, n_adapters=16, rank=16,
                  dtype=torch.bfloat16, device="cpu"):
    """The operator micro-benchmark: x ~ N(0,1), W ~ N(0,0.02), A ~ U(+-1/64),
    B ~ N(0,0.02), per-token ids uniform in [0, n_adapters), scale 2.0
    (shapes of ``tvm/lora_only/single_rank.py:66-103,142-155``).
    A is stored [N, r, in] and B [N, out, r] (peft's per-adapter layout)."""
    g = _gen(SEED_WEIGHTS, device)
    x = torch.randn(T, in_features, generator=g, device=device, dtype=torch.float32).to(dtype)
    W = (torch.randn(out_features, in_features, generator=g, device=device, dtype=torch.float32) * 0.02).to(dtype)
    A = ((torch.rand(n_adapters, rank, in_features, generator=g, device=device, dtype=torch.float32) * 2 - 1)
         / 64.0).to(dtype)
    B = (torch.randn(n_adapters, out_features, rank, generator=g, device=device, dtype=torch.float32) * 0.02).to(dtype)
    ids = torch.from_numpy(adapter_ids_uniform(T, n_adapters)).to(device)
    return dict(x=x, W=W, A=A, B=B, ids=ids, scale=2.0)
