"""Replay of a trace: given token ids, step by step, through the Decoder; logits to files.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Reads one JSON object a line from standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

entries: for each request its next tokens and the places among them whose logits are wanted;
end: requests that are finished after this step (their slot is free again).  For a step that
wants any, DIR/<step>.f32 receives little-endian float32 logits [wanted, vocab] in the order of
the entries; after every step a line "done <step>" is printed.  Nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


class SlotTable:
    """Which slot of the decoder each live request holds, and how many tokens it has consumed."""

    def __init__(self, n_slots: int):
        self.free = list(range(n_slots - 1, -1, -1))
        self.live = {}

    def slot(self, rid) -> int:
        if rid not in self.live:
            if not self.free:
                raise RuntimeError("more live requests than slots")
            self.live[rid] = [self.free.pop(), 0]
        return self.live[rid][0]

    def position(self, rid) -> int:
        return self.live[rid][1]

    def advance(self, rid, n: int) -> None:
        self.live[rid][1] += n

    def end(self, rid) -> None:
        if rid in self.live:
            self.free.append(self.live.pop(rid)[0])


def run(decoder, lines, out_dir: str, emit, slots: int) -> None:
    import torch
    table = SlotTable(slots)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        parts = []
        for e in step["entries"]:
            toks, want = e["tokens"], e["want"]
            if toks and not (0 <= min(toks) and max(toks) < decoder.vocab_size):
                raise ValueError(f"step {step['step']}: token id outside 0..{decoder.vocab_size - 1}")
            if not toks:
                continue
            slot = table.slot(e["id"])
            ids = torch.tensor(toks, dtype=torch.int32).to(decoder.device)
            logits = decoder.forward_logits(slot, ids, table.position(e["id"]), want)
            table.advance(e["id"], len(toks))
            if want:
                parts.append(logits)
        if parts:
            data = torch.cat(parts).cpu().numpy().astype("<f4").tobytes()
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(data)
        else:
            torch.cuda.synchronize()
        for rid in step.get("end", []):
            table.end(rid)
        emit(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--slots", type=int, default=4, help="most requests that are live at any time")
    a = ap.parse_args(argv)
    from . import build
    with _quiet_stdout():
        build.build()
    import torch  # noqa: F401

    from . import check_device_errors
    from .decoder import Decoder
    decoder = Decoder(a.model, dtype=a.dtype, max_batch=a.slots, max_seq_len=max(1, a.max_tokens))

    def emit(text):
        check_device_errors()
        print(text, flush=True)

    run(decoder, sys.stdin, a.out, emit, a.slots)
    decoder.close()
    return 0


class _quiet_stdout:
    """Compiler output goes to standard error: standard output carries the protocol."""

    def __enter__(self):
        sys.stdout.flush()
        self.saved = os.dup(1)
        os.dup2(2, 1)

    def __exit__(self, *exc):
        os.dup2(self.saved, 1)
        os.close(self.saved)


if __name__ == "__main__":
    sys.exit(main())
