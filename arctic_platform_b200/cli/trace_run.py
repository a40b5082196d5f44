"""Replays a trace of token ids through a served model and writes the logits it asks for.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  <  steps.jsonl

Every input line is one step: ``{"step": 0, "entries": [{"id": "a", "tokens": [...], "want": [...]}], "end": [...]}``.
All entries of a step run as ONE ragged batch of the engine's step function: each brings the next tokens of its request
(a portion of a prompt, or one decoded token); ``want`` are the places among them whose logits are written, in order, to
``OUT/<step>.f32`` (little-endian float32, ``[wanted, vocab]``).  Requests in ``end`` are finished after the step and
give their pages and state slot back.  After every step ``done <step>`` is printed.  The cache pool holds ``N`` tokens
(each live request rounded up to a page) and four requests.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import Dict

import numpy as np

MAX_LIVE = 4


def parse_args(argv=None) -> argparse.Namespace:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a token trace through a served model")
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=("bfloat16", "float32"))
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    return ap.parse_args(argv)


class Replay:
    """Request ids of a trace on an engine with the step interface (``open_sequence`` / ``step`` / ``close_sequence``)."""

    def __init__(self, engine, out_dir: Path):
        self.engine, self.out = engine, Path(out_dir)
        self.slots: Dict[str, int] = {}

    def run(self, rec: dict) -> None:
        work = []
        for e in rec["entries"]:
            if not e["tokens"]:
                continue
            if e["id"] not in self.slots:
                self.slots[e["id"]] = self.engine.open_sequence()
            work.append((self.slots[e["id"]], e["tokens"], e.get("want") or []))
        wanted = sum(len(w) for _, _, w in work)
        if work:
            logits = self.engine.step(work)
            if wanted:
                data = logits.float().cpu().numpy().astype("<f4", copy=False)
                np.ascontiguousarray(data).tofile(self.out / f"{rec['step']}.f32")
        for rid in rec.get("end") or []:
            if rid in self.slots:
                self.engine.close_sequence(self.slots.pop(rid))


def make_engine(model_dir: str, dtype: str, max_tokens: int):
    import torch
    from ..engine.stateful_sampler import StatefulSampler
    from ..models import registry
    from ..models.factory import LoaderContext, ModelSpec, build_model
    from ..ops import _lib
    spec = ModelSpec(model_dir, dtype=dtype)
    cfg = LoaderContext(spec).hf_config
    if not registry.is_stateful(cfg):
        raise SystemExit(f"{model_dir}: traces replay on the stateful engine ({', '.join(registry.architectures())})")
    if not torch.cuda.is_available():
        raise SystemExit("trace_run needs a CUDA device")
    _lib.serve_only(cfg.architecture)
    model = build_model(spec, device="cuda").model
    return StatefulSampler(cfg, "cuda", model=model, kv_cache_tokens=max_tokens, max_batch=MAX_LIVE,
                           max_seq_len=max(max_tokens, 64))


def main(argv=None) -> int:
    args = parse_args(argv)
    from ..ops import _lib
    engine = make_engine(args.model, args.dtype, args.max_tokens)
    replay = Replay(engine, args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        rec = json.loads(line)
        replay.run(rec)
        _lib.check_status(f"step {rec['step']}")
        print(f"done {rec['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
