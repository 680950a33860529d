#!/usr/bin/env python
"""Interactive text generation from a trained checkpoint.

Same flags as the reference REPL (generate.py:7-60).  ``--temperature 0`` decodes greedily and
``--top-k`` really filters.  A prompt can also be given with ``--prompt`` for non-interactive use.

``--model FOLDER`` loads any registered model (config.json and its weights; the configuration names the class) instead
of ``--config`` / ``--checkpoint``; ``--prompt-ids 5,17,3`` generates from token ids, without a tokenizer.
"""
from __future__ import annotations

import argparse
import os
import sys

import torch

ROOT = os.path.dirname(os.path.abspath(__file__))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

from llm_systems_from_scratch_b200.models.registry import load_model  # noqa: E402
from llm_systems_from_scratch_b200.models.transformer import TransformerLM  # noqa: E402
from llm_systems_from_scratch_b200.tokenizer.bpe import Tokenizer  # noqa: E402


def complete(model, tokenizer, prompt: str, device, max_tokens: int, temperature: float, top_k, eos_id):
    ids = torch.tensor([tokenizer.encode(prompt)], dtype=torch.long, device=device)
    out = model.generate(ids, max_new_tokens=max_tokens, temperature=temperature, top_k=top_k, eos_token_id=eos_id)
    return tokenizer.decode(out.reshape(-1).tolist())


def main(argv=None):
    ap = argparse.ArgumentParser(description="Generate text from a pretrained model")
    ap.add_argument("--config", type=str, default="model_config.json")
    ap.add_argument("--checkpoint", type=str, default="ckpt_final.pt")
    ap.add_argument("--model", type=str, default=None, help="model folder (config.json and weights) of any registered model")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16", help="with --model")
    ap.add_argument("--prompt-ids", type=str, default=None, help="token ids, with commas between them: print the ids that follow")
    ap.add_argument("--vocab", type=str, default="vocab.json")
    ap.add_argument("--merges", type=str, default="merges.json")
    ap.add_argument("--max-tokens", type=int, default=200)
    ap.add_argument("--temperature", type=float, default=1.0)
    ap.add_argument("--top-k", type=int, default=None)
    ap.add_argument("--device", type=str, default="auto")
    ap.add_argument("--prompt", type=str, default=None, help="generate once for this prompt and exit")
    args = ap.parse_args(argv)
    device = ("cuda" if torch.cuda.is_available() else "cpu") if args.device == "auto" else args.device
    if args.model is not None:
        model = load_model(args.model, getattr(torch, args.dtype), device)
    else:
        model = TransformerLM.from_pretrained(config_path=args.config, checkpoint_path=args.checkpoint).to(device)
    model.eval()
    if args.prompt_ids is not None:
        ids = torch.tensor([[int(t) for t in args.prompt_ids.split(",")]], dtype=torch.long, device=device)
        out = model.generate(ids, max_new_tokens=args.max_tokens, temperature=args.temperature, top_k=args.top_k)
        print(",".join(map(str, out.reshape(-1).tolist())))
        return
    tokenizer = Tokenizer.from_files(args.vocab, args.merges, special_tokens=["<|endoftext|>"])
    eos_id = tokenizer.encode("<|endoftext|>")[0]
    if args.prompt is not None:
        print(complete(model, tokenizer, args.prompt, device, args.max_tokens, args.temperature, args.top_k, eos_id))
        return
    print("Model loaded. Type your prompt (Ctrl+C to quit):\n")
    while True:
        try:
            prompt = input("> ")
        except (KeyboardInterrupt, EOFError):
            print()
            break
        if prompt:
            print(complete(model, tokenizer, prompt, device, args.max_tokens, args.temperature, args.top_k, eos_id))
            print()


if __name__ == "__main__":
    main()
