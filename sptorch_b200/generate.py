"""Generation from the command line: a model folder (config.json + model.safetensors) and token ids in, token ids out.

    python -m sptorch_b200.generate --model DIR --tokens 5,17,3 --max-new-tokens 32 [--top-k 1] [--temperature 1.0] ...

``--top-k 1`` (the default) is greedy.  The ids of the whole sequence are printed on one line, separated by commas."""
from __future__ import annotations

import argparse

import numpy as np

from .backend import BF16, F32, FfiBackend
from .registry import load_model


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="sptorch_b200.generate", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--tokens", required=True, help="token ids of the prompt, separated by commas")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--max-context", type=int, default=0, help="positions the cache holds (default: prompt + new tokens, or the model's own limit)")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--temperature", type=float, default=1.0)
    ap.add_argument("--top-k", type=int, default=1)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--repetition-penalty", type=float, default=1.0)
    ap.add_argument("--eos", type=int, default=None)
    ap.add_argument("--seed", type=int, default=None)
    a = ap.parse_args(argv)
    prompt = [int(t) for t in a.tokens.split(",") if t.strip()]
    rng = np.random.default_rng(a.seed)
    with FfiBackend.load() as b:
        model = load_model(b, a.model, seq_len=a.max_context or len(prompt) + a.max_new_tokens, dtype=BF16 if a.dtype == "bfloat16" else F32)
        try:
            out = model.generate(prompt, a.max_new_tokens, temperature=a.temperature, top_k=a.top_k, top_p=a.top_p, repetition_penalty=a.repetition_penalty,
                                 eos_token_id=a.eos, draw=rng.random)
        finally:
            model.close()
    print(",".join(str(t) for t in out))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
