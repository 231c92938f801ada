"""Replay a trace of given token ids through the engine and write the logits it asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

One JSON object a line: ``{"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}``. A step
feeds every entry's next tokens as ONE batch (:meth:`Engine.forward_tokens`: portions of prompts beside single decoded
tokens), continuing from the pages and recurrent states earlier steps left; ``want`` are places among an entry's tokens.
Wanted logits go to ``OUT/<step>.f32`` (little-endian fp32, [wanted, vocab]); requests in ``end`` give their pages and state
slot back. ``done <step>`` is printed after every step. Nothing is sampled.

``--max-tokens`` sizes the page pool (the most tokens live requests hold at any time); ``--max-requests`` the live requests,
which is also the number of recurrent-state slots.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path


def _family(model_dir: str) -> str:
    d = json.loads((Path(model_dir) / "config.json").read_text())
    return str(d.get("model_type") or d.get("architecture", "")).lower()


def load(model_dir: str, dtype: str, max_tokens: int, max_requests: int, device: str | None = None):
    import torch

    from ..api import LoadedModel, ModelLoadOptions
    from .kv_cache import PagedKVCache

    device = device or ("cuda" if torch.cuda.is_available() else "cpu")
    opt = ModelLoadOptions(device=device, dtype=getattr(torch, dtype), max_batch=max_requests, max_seq_len=max_tokens,
                           kv_pages=PagedKVCache.pages_for(max_tokens) + 1, state_slots=max_requests)
    return LoadedModel.load(model_dir, opt)


def replay(engine, lines, out_dir, emit) -> None:
    """Run the steps of ``lines`` (an iterable of JSON texts); ``emit(step)`` is called after each."""
    import numpy as np

    live: dict = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            seq = live.get(e["id"])
            if seq is None:
                seq = live[e["id"]] = engine.open_sequence()
            if e["tokens"]:
                entries.append((seq, e["tokens"], e["want"]))
        if entries:
            logits = engine.forward_tokens(entries)
            if logits.shape[0]:
                rows = logits.float().cpu().numpy().astype("<f4")
                Path(out_dir, f"{step['step']}.f32").write_bytes(np.ascontiguousarray(rows).tobytes())
        for rid in step.get("end", []):
            seq = live.pop(rid, None)
            if seq is not None:
                engine.release(seq)
        if engine.cuda:
            from ..ops import native

            native.check_status(engine.device)
        emit(step["step"])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a token trace and write the wanted logits")
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the page pool holds")
    ap.add_argument("--max-requests", type=int, default=4, help="live requests (recurrent-state slots)")
    ap.add_argument("--device", default=None, help="cuda (default where there is one) or cpu")
    a = ap.parse_args(argv)
    from .. import build
    from ..ops import native

    library = build.ensure_family(_family(a.model))
    native.use_library(library)
    engine = load(a.model, a.dtype, a.max_tokens, a.max_requests, a.device).engine

    def emit(step):
        print(f"done {step}", flush=True)

    replay(engine, sys.stdin, a.out, emit)
    return 0
