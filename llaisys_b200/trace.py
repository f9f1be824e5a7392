"""Trace replay: runs recorded token ids through a model with the engine's own batched steps and cache, and writes logits
at chosen positions. No sampling; comparing two builds, two precisions or two ways of cutting the same prompts is what it is
for.

One step per line of standard input:
    {"step": 3, "entries": [{"id": "r1", "tokens": [8, 2], "want": [1]}, ...], "end": ["r0"]}
An id that is new takes a sequence (and its state slot); ids under "end" return theirs once the step has run. "want" holds
indices into that entry's tokens. Logits go to <out>/<step>.f32, raw little-endian float32, one row of the vocabulary per
wanted token; "done <step>" follows on standard output.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

MAX_LIVE = 4  # state slots


class TraceRunner:
    """The live requests of a trace on one model."""

    def __init__(self, model, max_tokens: int):
        self.model = model
        model.configure_cache(MAX_LIVE, max_tokens, max_tokens)
        self._seq: dict[str, int] = {}

    def step(self, entries: list[dict], end: list[str] = ()):
        """-> logits [wanted, vocab]"""
        seqs, tokens, rows, at = [], [], [], 0
        for e in entries:
            if not e["tokens"]:
                continue
            if e["id"] not in self._seq:
                self._seq[e["id"]] = self.model.add_seq()
            seqs.append(self._seq[e["id"]])
            tokens.append(e["tokens"])
            rows += [at + w for w in e.get("want", ())]
            at += len(e["tokens"])
        logits = self.model.step_rows(seqs, tokens, rows) if seqs else None
        for rid in end:
            if rid in self._seq:
                self.model.free_seq(self._seq.pop(rid))
        return logits


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at most")
    args = ap.parse_args(argv)

    from .models import load_model
    from .models.base import DTYPE_NAMES

    runner = TraceRunner(load_model(args.model, dtype=DTYPE_NAMES[args.dtype]), args.max_tokens)
    out = Path(args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        msg = json.loads(line)
        logits = runner.step(msg.get("entries", []), msg.get("end", []))
        if logits is not None and logits.shape[0]:
            logits.astype("<f4").tofile(out / f"{msg['step']}.f32")
        print(f"done {msg['step']}", flush=True)
    return 0
