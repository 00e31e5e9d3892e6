"""`bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N`: replay recorded requests.

Steps come on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step are one batch of the engine (LLMEngine.replay_step): portions of prompts beside single decoded
tokens, from the paged cache and the state slots earlier steps left.  A request is admitted at its first entry, may be
left out of steps, and gives its blocks and its slot back at `end`.  When a step asks for logits they are written to
OUT/<step>.f32 (little-endian fp32, [wanted, vocab], in the order of the entries); `done <step>` follows every step.
`--max-tokens` sizes the cache pool: the most tokens that live requests hold at any time.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def build_engine(model: str, dtype: str, max_tokens: int, device: str = "auto", max_live: int = 4, block_size: int = 16):
    from .engine.llm_engine import EngineConfig, LLMEngine
    from .models import load_model_args
    from .models.registry import kernel_sources_of
    from .ops import _lib
    _lib.select_sources(kernel_sources_of(load_model_args(model)))
    blocks = -(-max_tokens // block_size)
    tokens = blocks * block_size
    return LLMEngine(EngineConfig(
        model=model, dtype=dtype, device=device, block_size=block_size, num_blocks=blocks + 1,      # block 0 is padding
        max_seqs_per_batch=max_live, max_running_seqs=max_live, max_tokens_per_batch=tokens, max_model_len=tokens,
        max_sample_rows=tokens, enable_prefix_cache=False))


def run(engine, lines, out_dir: str, echo):
    import numpy as np
    for line in lines:
        line = line.strip()
        if not line:
            continue
        step = json.loads(line)
        if step.get("entries"):
            logits = engine.replay_step([(e["id"], e["tokens"], e.get("want") or []) for e in step["entries"]])
            if logits.shape[0]:
                logits.numpy().astype("<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
                assert np.isfinite(logits.numpy()).all(), "logits are not finite"
        for rid in step.get("end") or []:
            engine.replay_end(rid)
        echo(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay recorded requests and write their logits.")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    ap.add_argument("--device", default="auto")
    a = ap.parse_args(argv)

    def echo(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    run(build_engine(a.model, a.dtype, a.max_tokens, a.device), sys.stdin, a.out, echo)
    return 0
