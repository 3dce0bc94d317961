"""Greedy generation from the command line, for any model of the registry (models.py):

    python -m ternary_llm_b200.generate --model PATH --tokens 5,17,3 --steps 32 [--dtype float32]

PATH is a .tllm file or a folder with config.json and model.safetensors.  Token ids in, token
ids out (there is no tokenizer here): the prompt runs through Decoder.forward, the rest through
Decoder.generate, which replays one captured step per token.
"""
from __future__ import annotations

import argparse
import sys


def parse_tokens(text: str):
    try:
        toks = [int(v) for v in text.replace(",", " ").split()]
    except ValueError:
        raise argparse.ArgumentTypeError(f"{text!r}: token ids are integers separated by commas")
    if not toks or min(toks) < 0:
        raise argparse.ArgumentTypeError(f"{text!r}: at least one non-negative token id")
    return toks


def greedy(decoder, prompt, n_steps: int):
    """The n_steps tokens that follow the prompt, and milliseconds per replayed step (None for one)."""
    import torch
    if max(prompt) >= decoder.vocab_size:
        raise ValueError(f"token id {max(prompt)} outside the vocabulary of {decoder.vocab_size}")
    logits = decoder.forward(torch.tensor(prompt, dtype=torch.int32).to(decoder.device), 0)
    first = int(logits.float().argmax().item())
    if n_steps <= 1:
        return [first][:n_steps], None
    rest, ms = decoder.generate(first, len(prompt), n_steps - 1)
    return [first] + rest, ms


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m ternary_llm_b200.generate", description="Greedy generation on token ids.")
    ap.add_argument("--model", required=True, help=".tllm file, or folder with config.json and model.safetensors")
    ap.add_argument("--tokens", required=True, type=parse_tokens, help="prompt token ids, separated by commas")
    ap.add_argument("--steps", type=int, default=32, help="tokens to generate")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"], help="models of mixer layers only")
    a = ap.parse_args(argv)
    from . import build
    build.build()
    from .decoder import Decoder
    decoder = Decoder(a.model, dtype=a.dtype, max_seq_len=len(a.tokens) + a.steps + 1)
    out, ms = greedy(decoder, a.tokens, a.steps)
    print(",".join(map(str, out)))
    if ms is not None:
        print(f"{ms:.3f} ms per token", file=sys.stderr)
    decoder.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
