"""Trace runner: feeds given token ids through a model step by step and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input carries one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step are one batch of the engine (:meth:`Engine.feed`): portions of prompts beside single tokens, each run
from what earlier steps left in the cache. A request is admitted at its first entry and its blocks return to the pool after
the step that names it in ``end``. A step with wanted places writes ``DIR/<step>.f32`` (little-endian 32-bit floats, [wanted,
vocab], in the order of the entries); after every step ``done <step>`` goes to standard output. The KV pool holds N tokens
(rounded up to blocks) and at most ``LIVE_REQUESTS`` requests are live.

Exit codes: 0 at the end of the input, 2 on unusable input or without a GPU, 3 when the model has no 32-bit form.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

LIVE_REQUESTS = 4


class TraceError(RuntimeError):
    pass


class TraceRunner:
    """Requests by name on top of an engine whose forward takes mixed batches."""

    def __init__(self, engine, vocab: int):
        self.engine, self.vocab = engine, vocab
        self.live: dict[str, object] = {}

    def step(self, entries: list[dict], end: list[str]):
        """Run one step; returns the wanted logits [wanted, vocab] as FP32 on the host, or None."""
        from ..engine.engine import Span
        spans = []
        for e in entries:
            tokens = [int(t) for t in e["tokens"]]
            if not tokens or any(not 0 <= t < self.vocab for t in tokens):
                raise TraceError(f"request {e['id']}: no tokens, or a token outside the vocabulary")
            if any(not 0 <= int(k) < len(tokens) for k in e.get("want", [])):
                raise TraceError(f"request {e['id']}: a wanted place outside the entry")
            seq = self.live.get(e["id"])
            if seq is None:
                if len(self.live) >= LIVE_REQUESTS:
                    raise TraceError(f"more than {LIVE_REQUESTS} live requests")
                seq = self.live[e["id"]] = self.engine.add_sequence(tokens)
            spans.append(Span(seq, tokens, [int(k) for k in e.get("want", [])]))
        logits = self.engine.feed(spans) if spans else None
        out = None if logits is None else logits.float().cpu().contiguous()
        for name in end:
            seq = self.live.pop(name, None)
            if seq is None:
                raise TraceError(f"request {name} is not live")
            self.engine.free_sequence(seq.seq_id)
        return out


def load_engine(model_dir: str, dtype: str, max_tokens: int, device: str = "cuda:0"):
    """(model, engine) with a KV pool of ``max_tokens`` tokens."""
    from ..api import Model
    from ..config import Settings
    block = Settings().kv_block
    pool = (max_tokens + block - 1) // block * block
    model = Model.load(model_dir, Settings(capacity=pool, kv_tokens=pool, max_batch=LIVE_REQUESTS, dtype=dtype), device=device)
    if not model.engine.mixed_batches:
        raise TraceError(f"{model.spec.arch}: the model's forward does not take mixed batches")
    return model, model.engine


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], required=True)
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    a = ap.parse_args(argv)
    import torch
    if not torch.cuda.is_available():
        sys.stderr.write("trace_run needs a CUDA device\n")
        return 2
    from ..config import GPU_FP32_ARCHS, read_model_spec
    from ..ops import lib
    spec = read_model_spec(a.model)
    lib.restrict_to(spec.arch)
    dtype = {"bfloat16": "bf16", "float32": "fp32"}[a.dtype]
    if dtype == "fp32" and spec.arch not in GPU_FP32_ARCHS:
        sys.stderr.write(f"{spec.arch} has no 32-bit form\n")
        return 3
    model, engine = load_engine(a.model, dtype, a.max_tokens)
    runner = TraceRunner(engine, model.spec.vocab)
    out = Path(a.out)
    try:
        for line in sys.stdin:
            if not line.strip():
                continue
            req = json.loads(line)
            logits = runner.step(req.get("entries", []), req.get("end", []))
            if logits is not None:
                (out / f"{int(req['step'])}.f32").write_bytes(logits.numpy().astype("<f4").tobytes())
            print(f"done {req['step']}", flush=True)
    except (TraceError, json.JSONDecodeError, KeyError) as e:
        sys.stderr.write(f"{type(e).__name__}: {e}\n")
        return 2
    return 0
