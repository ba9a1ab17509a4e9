"""Teacher-forced replay: feeds given token ids through the engine, step by step, and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Standard input holds one step per line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

All entries of a step run as one batch (:meth:`~mfq_b200.engine.llm_engine.LLMEngine.extend`), each from where its request
stood; ``want`` are places among the entry's tokens, ``end`` the requests whose pages and row are given back after the step.
For a step that wants something, ``<out>/<step>.f32`` gets the logits in the order of the entries and of ``want`` (little-endian
fp32, ``[wanted, vocabulary]``).  After every step the line ``done <step>`` is printed.  ``--max-tokens`` sizes the KV pool: what
the live requests hold at any time, each rounded up to a multiple of 64.

Exit codes: 0 at the end of the input, 3 when the model's family does not run in the requested element type.  The CUDA
libraries the family needs are compiled first if they are missing or out of date.
"""

from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

MAX_REQUESTS = 4


def parse_args(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="replay tokens through a model and write logits")
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    return ap.parse_args(argv)


class Replay:
    """Request names on top of an engine's batch rows."""

    def __init__(self, engine) -> None:
        self.engine = engine
        self.rows: dict[str, int] = {}

    def _row(self, name: str) -> int:
        if name not in self.rows:
            free = [r for r in range(self.engine.max_batch) if r not in self.rows.values()]
            if not free:
                raise RuntimeError(f"more than {self.engine.max_batch} live requests")
            self.engine.open_row(free[0])
            self.rows[name] = free[0]
        return self.rows[name]

    def step(self, doc: dict):
        """Run one step; the logits it wants as an fp32 numpy array, or None."""
        entries = [e for e in doc["entries"] if e["tokens"]]
        portions = [(self._row(e["id"]), e["tokens"]) for e in entries]
        logits = self.engine.extend(portions, [e.get("want", ()) for e in entries]) if portions else None
        for name in doc.get("end", ()):
            if name in self.rows:
                self.engine.release(self.rows.pop(name))
        return None if logits is None else logits.float().cpu().numpy().astype("<f4")


def run(engine, lines, out: Path, emit) -> None:
    import torch

    from .. import ops
    replay = Replay(engine)
    for line in lines:
        if not line.strip():
            continue
        doc = json.loads(line)
        logits = replay.step(doc)
        if engine.device.type == "cuda":
            torch.cuda.synchronize()
            ops.Workspace.get(engine.device).check()
        if logits is not None:
            logits.tofile(out / f"{int(doc['step'])}.f32")
        emit(f"done {int(doc['step'])}")


def main(argv=None) -> int:
    args = parse_args(argv)
    from ..architectures import config_from_hf
    from ..models import registry
    family = registry.find(config_from_hf(json.loads((Path(args.model) / "config.json").read_text())))
    dtype = args.dtype if args.dtype in family.dtypes else "auto"
    if args.dtype == "float32" and dtype == "auto":
        print(f"models of the {family.name} family do not run in float32", file=sys.stderr)
        return 3
    from ..ops.build import build
    for library in family.kernels:
        build(only=library)
    from ..checkpoint import load_engine
    from .kv_cache import PAGE_SIZE
    pages = -(-args.max_tokens // PAGE_SIZE)
    engine, _tokenizer, _cfg = load_engine(args.model, "cuda", max_batch=MAX_REQUESTS, max_seq_len=pages * PAGE_SIZE,
                                           num_pages=pages + 1, use_graphs=False, dtype=dtype)
    run(engine, sys.stdin, Path(args.out), lambda text: print(text, flush=True))
    return 0
