"""Replays a trace: steps of given token ids through a model's own step functions, logits of the wanted places into files.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR [--max-tokens N]

Standard input holds one JSON object a line: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  A request's first entry
starts its sequence, later ones continue it from the cache and state (portions of any size); "end" gives back what it holds.  One
request is in flight at a time.  A step with wanted places writes OUT/<step>.f32, [wanted, vocab] little-endian f32; every step is
answered with the line "done <step>"."""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

from .backend import BF16, F32, FfiBackend, HalError, bf16_bits_to_f32
from .registry import load_model


class Replay:
    def __init__(self, model):
        self.model, self.live = model, None
        model.enable_kv_cache()

    def feed(self, request, tokens, want) -> np.ndarray:
        """Runs the request's next tokens; logits [len(want), vocab] of the wanted places."""
        m = self.model
        if self.live is None:
            m.reset_cache()
            self.live = request
        elif self.live != request:
            raise HalError(f"request {request!r} cannot start before {self.live!r} has ended: one sequence is in flight at a time")
        if not tokens:
            return np.empty((0, m.cfg["vocab"]), np.float32)
        d_log = m.extend_device(np.asarray(tokens).reshape(1, -1))
        return m.read_logit_rows(d_log, want)

    def end(self, request):
        if self.live == request:
            self.live = None
            self.model.reset_cache()


def replay(model, lines, out_dir: str, answer) -> None:
    r = Replay(model)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        parts = [r.feed(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]]
        rows = np.concatenate(parts) if parts else np.empty((0, 0), np.float32)
        if rows.size:
            part = os.path.join(out_dir, f".{step['step']}.part")
            rows.astype("<f4").tofile(part)
            os.replace(part, os.path.join(out_dir, f"{step['step']}.f32"))
        for request in step.get("end", []):
            r.end(request)
        answer(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, default=0, help="the most tokens live requests hold at any time (sizes the cache)")
    a = ap.parse_args(argv)
    with FfiBackend.load() as b:
        model = load_model(b, a.model, seq_len=a.max_tokens, dtype=BF16 if a.dtype == "bfloat16" else F32)
        try:
            replay(model, sys.stdin, a.out, lambda text: print(text, flush=True))
        finally:
            model.close()
    return 0
