"""Command line of the framework.

    generate --model DIR --prompt "3 17 5" [--prompt ...] [--max-new-tokens N] [--eos ID] [--dtype ...]
        greedy generation through the auto-batcher; prompts and answers are token ids, one answer a line
    replay --model DIR --dtype ... --out DIR --max-tokens N
        feeds the token ids of JSON steps on standard input and writes logits (see ``replay``; also ``bin/trace_run``)
"""
from __future__ import annotations

import argparse

DTYPES = ("bfloat16", "float32")


class TokenIds:
    """Tokenizer of prompts that are token ids already."""

    def __init__(self, eos_token_id=None):
        self.eos_token_id = eos_token_id

    def __call__(self, prompt, return_tensors="pt"):
        import torch
        return {"input_ids": torch.tensor([list(prompt)], dtype=torch.long)}

    def decode(self, ids):
        return [int(i) for i in ids]


def add_replay_arguments(ap):
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=DTYPES, default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")


def generate(args) -> int:
    import torch

    from . import auto_batcher, build, registry
    build.build()
    prompts = [[int(t) for t in p.replace(",", " ").split()] for p in args.prompt]
    ab = auto_batcher.LlamaAutoBatcherClass()
    try:
        ab.set_model_dir(args.model, dtype=getattr(torch, args.dtype))
    except registry.UnsupportedPrecision as e:
        raise SystemExit(str(e))
    ab.set_tokenizer(TokenIds(args.eos))
    ab.set_exec_config(auto_batcher.LlamaExecConfig(max(len(p) for p in prompts), args.max_new_tokens, args.page_size))
    answers = [ab.generate(ab.create_var(p)) for p in prompts]
    ab.compile()
    ab.execute()
    for a in answers:
        print(" ".join(str(t) for t in a.var))
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="b200-multilora", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy generation, prompts as token ids")
    g.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    g.add_argument("--prompt", action="append", required=True, help="token ids separated by blanks or commas (repeatable)")
    g.add_argument("--max-new-tokens", type=int, default=32)
    g.add_argument("--eos", type=int, default=None, help="token id that ends an answer")
    g.add_argument("--page-size", type=int, default=16, choices=(16, 32))
    g.add_argument("--dtype", choices=DTYPES, default="bfloat16")
    add_replay_arguments(sub.add_parser("replay", help="feed given tokens step by step, write logits"))
    args = ap.parse_args(argv)
    if args.command == "replay":
        from . import replay
        return replay.main(args)
    return generate(args)
