"""Trace replay: feed given token ids through the serving engine step by step and write the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come from standard input, one JSON object a line:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}
All entries of a step are one batch of the engine (LLMEngine.replay_step). Wanted logits go to <out>/<step>.f32 as
little-endian fp32 [wanted, vocab]; "done <step>" is printed after every step. Requests in "end" give their pages and
state slot back. Exit code 3: the model's family has no kernels for that dtype."""
from __future__ import annotations

import argparse
import json
import os
import sys

MAX_LIVE = 4                 # requests alive at any time: state slots of the replay engine


def build_engine(model: str, dtype_name: str, max_tokens: int, device: str = "cuda", block_size: int = 16):
    import torch

    from ..models.config import resolve_config
    from ..models.registry import family_of
    from .engine import LLMEngine
    from .model_runner import TPContext
    from .tokenizer import ByteTokenizer

    dtype = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype_name]
    cfg = resolve_config(model)
    fam = family_of(cfg)
    if device == "cuda" and dtype not in fam.dtypes:
        print(f"{fam.name} has no {dtype_name} kernels", file=sys.stderr)
        sys.exit(3)
    w = fam.load_weights(cfg, model, device, dtype)
    n = -(-max_tokens // 64) * 64
    return LLMEngine(cfg, w, TPContext(), ByteTokenizer(cfg.vocab_size), block_size=block_size, num_blocks=n // block_size,
                     max_num_seqs=MAX_LIVE, max_num_batched_tokens=n, max_model_len=n, async_scheduling=False)


def run(engine, lines, out_dir: str, emit) -> None:
    import numpy as np

    from .params import Request, SamplingParams

    live: dict[str, Request] = {}
    for line in lines:
        if not line.strip():
            continue
        st = json.loads(line)
        entries = []
        for e in st["entries"]:
            r = live.get(e["id"])
            if r is None:
                r = live[e["id"]] = Request(e["id"], [], SamplingParams(temperature=0.0))
            entries.append((r, list(e["tokens"]), list(e["want"])))
        logits = engine.replay_step(entries) if entries else None
        if logits is not None:
            np.ascontiguousarray(logits.numpy(), dtype="<f4").tofile(os.path.join(out_dir, f"{st['step']}.f32"))
        for rid in st.get("end", []):
            engine.replay_end(live.pop(rid))
        emit(f"done {st['step']}")


def main(argv=None) -> None:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="size of the cache pool: tokens of all live requests")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"], help=argparse.SUPPRESS)
    a = ap.parse_args(argv)
    os.makedirs(a.out, exist_ok=True)
    eng = build_engine(a.model, a.dtype, a.max_tokens, a.device)
    run(eng, sys.stdin, a.out, lambda s: print(s, flush=True))


if __name__ == "__main__":
    main()
