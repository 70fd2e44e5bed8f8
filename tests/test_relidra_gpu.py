"""Relidra through the framework: engine, cache, batches, portions, captured decoding, scheduler, command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import relidra_cases as rc
from conftest import PKG, ROOT, load
from oracle import relidra as orl

pytestmark = pytest.mark.gpu

BF, F32 = torch.bfloat16, torch.float32
_cache = {}


def case(name, dtype, cuda):
    key = (name, dtype)
    if key not in _cache:
        cfg = rc.CONFIGS[name]
        p = rc.weights(cfg)
        _cache[key] = (cfg, load("registry").build_model(cfg, p, device=cuda, dtype=dtype), orl.OracleRelidra(cfg, p))
    return _cache[key]


def serve(model, max_batch=4, total=1024, rows=256, page=16):
    kv = model.new_cache(max_batch, total, rows, page)
    return kv, model.new_engine(kv, rows)


def alone(model, toks, want=None, rows=256, page=16):
    kv, eng = serve(model, 1, len(toks) + 1, rows, page)
    kv.add_sequence(0)
    return eng.extend([0], [toks], want=[list(range(len(toks))) if want is None else want])[0].cpu()


NAMES = sorted(rc.CONFIGS)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_match_the_oracle(cuda, name, dtype):
    cfg, model, oracle = case(name, dtype, cuda)
    for n in (1, 2, 17, 150):
        toks = rc.tokens(cfg, n, n)
        want = oracle.forward(toks)[0]
        rc.check(alone(model, toks), want, dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("name", NAMES)
def test_prefill_against_decoding_token_by_token(cuda, name, dtype):
    """Every position decoded alone from the cache, across page borders, agrees with the prompt pass and the oracle."""
    cfg, model, oracle = case(name, dtype, cuda)
    toks = rc.tokens(cfg, 40, 5)
    kv, eng = serve(model)
    kv.add_sequence(7)
    got = [eng.extend([7], [toks[:1]])[0][0].cpu()]
    for t in toks[1:]:
        got.append(eng.decode([7], [t], [-1])[0][0].cpu().clone())
    want = oracle.forward(toks)[0]
    rc.check(torch.stack(got), want, dtype)
    rc.check(torch.stack(got), alone(model, toks), dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("cuts", [[2] * 20, [3, 37, 2, 16, 17, 1, 30, 2], [15, 2, 15, 2, 94], [128, 2, 1, 125], [255, 2, 3]])
def test_portions_of_prompts(cuda, dtype, cuts):
    """Cut anywhere, down to two tokens, small passes included: the logits of every position stay the same."""
    for name in ("odd", "deep", "streams"):
        cfg, model, oracle = case(name, dtype, cuda)
        toks = rc.tokens(cfg, sum(cuts), len(cuts))
        want = oracle.forward(toks)[0]
        for rows in (256, 24):
            kv, eng = serve(model, rows=rows)
            kv.add_sequence(0)
            got, a = [], 0
            for n in cuts:
                got.append(eng.extend([0], [toks[a:a + n]], want=[list(range(n))])[0].cpu())
                a += n
            rc.check(torch.cat(got), want, dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_unequal_requests_in_one_batch(cuda, name, dtype):
    """Prompts of different lengths in shared passes, then shared decode steps with different contexts."""
    cfg, model, oracle = case(name, dtype, cuda)
    prompts = [rc.tokens(cfg, n, 20 + n) for n in (1, 33, 90, 16)]
    kv, eng = serve(model, rows=64)
    for s in range(4):
        kv.add_sequence(s)
    want_rows = [[0], [0, 15, 16, 32], [89], [15]]
    got = eng.extend([0, 1, 2, 3], prompts, want=want_rows)[0].cpu()
    rc.check(got, torch.cat([oracle.forward(p)[0][w] for p, w in zip(prompts, want_rows)]), dtype)
    nxt = [rc.tokens(cfg, 5, 40 + s) for s in range(4)]
    for k in range(5):
        order = [2, 0, 3, 1] if k % 2 else [0, 1, 2, 3]
        got = eng.decode(order, [nxt[s][k] for s in order], [-1] * 4)[0].cpu()
        rc.check(got, torch.stack([oracle.forward(prompts[s] + nxt[s][:k + 1])[0][-1] for s in order]), dtype)


def test_pages_and_slots_used_again(cuda):
    """Sequences that end give their pages back; whoever gets them next -- shorter, longer, interleaved with a survivor --
    sees none of the old contents."""
    cfg, model, oracle = case("odd", F32, cuda)
    kv, eng = serve(model, max_batch=2, total=160, rows=64)
    keep = rc.tokens(cfg, 50, 1)
    kv.add_sequence(100)
    eng.extend([100], [keep[:20]])
    at = 20
    for r, n in enumerate((60, 3, 17, 90, 1, 33)):
        toks = rc.tokens(cfg, n, 60 + r)
        kv.add_sequence(r)
        got = eng.extend([r], [toks], want=[list(range(n))])[0].cpu()
        rc.check(got, oracle.forward(toks)[0], F32)
        got = eng.extend([100], [keep[at:at + 5]], want=[[0, 4]])[0].cpu()
        rc.check(got, oracle.forward(keep[:at + 5])[0][[at, at + 4]], F32)
        at += 5
        kv.remove_sequence(r)
    assert len(kv._free) == kv.n_pages - kv._n_pages_of[100]


def test_stale_values_in_reused_memory_do_not_leak(cuda):
    """Everything a new sequence has not written is NaN: cache pages and the engine's buffers."""
    for dtype in (BF, F32):
        cfg, model, oracle = case("deep", dtype, cuda)
        kv, eng = serve(model)
        for t in [*kv.pages.values(), *(t for e in kv.states.values() for t in e.values())]:
            t.fill_(float("nan"))
        for name in ("proj", "mixed", "q", "act", "xn", "y", "emb", "streams"):
            getattr(eng, name).fill_(float("nan"))
        toks = rc.tokens(cfg, 37, 9)
        kv.add_sequence(0)
        got = [eng.extend([0], [toks[:20]], want=[list(range(20))])[0].cpu()]
        got += [eng.decode([0], [t], [-1])[0].cpu().clone() for t in toks[20:]]
        want = oracle.forward(toks)[0]
        rc.check(torch.cat(got), want, dtype)


def test_cache_entries_follow_the_runs(cuda):
    """Every run of a looped layer has pages or a state of its own; keys and values are what the oracle's first layer makes."""
    cfg, model, oracle = case("deep", F32, cuda)
    kv, eng = serve(model)
    assert sorted(kv.pages) == [1, 3, 5] and sorted(kv.states) == [0, 2, 4]
    assert kv.state(0, "S").dtype == F32 and len({kv.state(e, "S").data_ptr() for e in (0, 2, 4)}) == 3
    cfg, model, oracle = case("wide", F32, cuda)
    kv, eng = serve(model)
    kv.add_sequence(3)
    toks = rc.tokens(cfg, 35, 2)
    eng.extend([3], [toks])
    p, m = oracle.p, cfg["layers"][0]["mixer"]
    u = p["l0.hc1.in"][0] * p["embed"][torch.tensor(toks)]
    v = (orl.layer_norm(u, p["l0.norm1"], cfg["norm"]["eps"]) @ p["l0.mix.k"].T + p["l0.mix.k.b"]).view(35, m["kv_heads"], m["dim"])
    k = orl.rms(orl.rotate(v, torch.arange(35), m["rot"]["dims"], m["rot"]["base"], 1.0), cfg["norm"]["eps"])
    for got, want in zip(kv.gather(3, 0), (k, v)):
        torch.testing.assert_close(got.double().cpu(), want, atol=1e-4, rtol=1e-4)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_captured_decode_steps(cuda, dtype):
    """A CUDA graph of the whole step, long enough to cross pages and attention blocks; the oracle scores every step."""
    cfg, model, oracle = case("deep", dtype, cuda)
    n = 150
    kv, eng = serve(model, max_batch=3, total=1200)
    prompts = [rc.tokens(cfg, k, k) for k in (5, 16, 60)]
    for s in range(3):
        kv.add_sequence(s)
    _, first = eng.prefill([0, 1, 2], prompts, [-1] * 3)
    g = eng.capture_decode([0, 1, 2], [-1] * 3, reserve_tokens=n)
    eng.tokens[:3].copy_(first)
    toks, logits = [first.tolist()], []
    for _ in range(n):
        g.replay()
        logits.append(eng.logits[:3].cpu().clone())
        toks.append(eng.next_tok[:3].tolist())
    eng.check_status()
    for s in range(3):
        gen = [t[s] for t in toks]
        n0 = len(prompts[s])
        want = oracle.forward(prompts[s] + gen[:-1])[0][n0:]
        rc.check(torch.stack([l[s] for l in logits]), want, dtype)


def _save(tmp_path, name):
    from safetensors.torch import save_file
    cfg = rc.CONFIGS[name]
    d = str(tmp_path / name)
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(rc.weights(cfg), os.path.join(d, "model.safetensors"))
    return cfg, d


@pytest.mark.parametrize("device_loop", [True, False])
def test_greedy_generation_through_the_scheduler(cuda, tmp_path, device_loop):
    """The auto-batcher on a model folder: unequal prompts and lengths, one fused decode node, tokens of the oracle."""
    ab, cli = load("auto_batcher"), load("cli")
    cfg, d = _save(tmp_path, "odd")
    oracle = orl.OracleRelidra(cfg, rc.weights(cfg))
    b = ab.LlamaAutoBatcherClass()
    b.set_model_dir(d, dtype=F32)
    b.set_tokenizer(cli.TokenIds())
    b.set_exec_config(ab.LlamaExecConfig(max_prompt_len=40, max_gen_len=20, page_size=16))
    prompts, lens = [rc.tokens(cfg, n, n) for n in (3, 40, 16, 1)], [20, 7, 18, 4]
    out = [b.generate(b.create_var(p), n) for p, n in zip(prompts, lens)]
    b.compile()
    b.graph.device_loop = device_loop
    b.execute()
    for v, p, n in zip(out, prompts, lens):
        assert list(v.var) == oracle.greedy(p, n)[0]


def test_command_line_generates(cuda, tmp_path):
    cfg, d = _save(tmp_path, "deep")
    oracle = orl.OracleRelidra(cfg, rc.weights(cfg))
    prompts = [rc.tokens(cfg, 4, 1), rc.tokens(cfg, 9, 2)]
    cmd = [sys.executable, "-m", PKG, "generate", "--model", d, "--max-new-tokens", "6", "--dtype", "float32"]
    for p in prompts:
        cmd += ["--prompt", " ".join(map(str, p))]
    r = subprocess.run(cmd, cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = [[int(t) for t in line.split()] for line in r.stdout.strip().splitlines()[-2:]]
    assert got == [oracle.greedy(p, 6)[0] for p in prompts]


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(cuda, tmp_path, dtype):
    """Steps on standard input, logits in files; requests that end and come again; a step that wants nothing."""
    cfg, d = _save(tmp_path, "odd")
    oracle = orl.OracleRelidra(cfg, rc.weights(cfg))
    a, b = rc.tokens(cfg, 45, 1), rc.tokens(cfg, 20, 2)
    steps = [
        ([("a", a[:17], [0, 16])], []), ([("a", a[17:19], [])], []), ([("a", a[19:20], [0]), ("b", b[:18], [17])], []),
        ([("b", b[18:19], [0]), ("a", a[20:21], [0])], []), ([("a", a[21:], [23, 0])], ["a"]), ([("b", b[19:], [0])], ["b"]),
        ([("a", b, [3, 19])], ["a"]),
    ]
    lines = [json.dumps({"step": i, "entries": [{"id": n, "tokens": t, "want": w} for n, t, w in e], "end": end})
             for i, (e, end) in enumerate(steps)]
    out = str(tmp_path / "out")
    os.makedirs(out)
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", out, "--max-tokens", "80"],
                       input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    full = {n: oracle.forward(t)[0] for n, t in (("a", a), ("b", b))}
    at = {"a": 0, "b": 0}
    for i, (e, end) in enumerate(steps):
        want = []
        for n, t, w in e:
            ref = full["b" if i == 6 else n]
            want += [ref[at[n] + k] for k in w]
            at[n] += len(t)
        at.update({n: 0 for n in end})
        path = os.path.join(out, f"{i}.f32")
        assert os.path.exists(path) == bool(want)
        if want:
            got = torch.from_numpy(np.fromfile(path, dtype="<f4")).view(len(want), cfg["vocab"])
            rc.check(got, torch.stack(want), getattr(torch, dtype))
