"""Trace runner: feeds given token ids through a served model step by step and writes logits; nothing is
sampled.  It drives the serving engine's own step over its pages and state slots.

Input, one JSON object a line::

    {"step": 7, "entries": [{"id": "q1", "tokens": [11, 42], "want": [1]}], "end": ["q0"]}

All entries of a step run as one batch: the next tokens of each request (a portion of a prompt or one
decoded token), with the logits asked for at ``want`` (places among these tokens).  ``end`` lists requests
that are over after the step; their pages and state slot are given back.  A step that wants something
writes ``<out>/<step>.f32``: little-endian fp32 [wanted, vocab] in the order of the entries and of ``want``.
``done <step>`` on standard output follows every step.

Exit codes: 0 the input ended, 2 bad arguments or input."""
from __future__ import annotations

import argparse
import json
import os
import sys

#: live requests at any time (state slots)
MAX_LIVE = 4
#: a request's token count is rounded up to this many in ``--max-tokens``
ROUND = 64


class TraceSession:
    """Requests fed portion by portion into an engine that offers ``step_logits``."""

    def __init__(self, engine):
        from .paged import BlockAllocator, StateSlots
        self.engine = engine
        self.alloc = BlockAllocator(engine.num_blocks, engine.block_size)
        self.slots = StateSlots(engine.state_slots) if engine.state_slots else None
        self.live = {}

    def step(self, entries):
        """``entries``: (id, tokens, want) -> fp32 logits [wanted, vocab] (numpy) or None."""
        import numpy as np
        from .hybrid import Entry
        from .paged import CachedSequence
        batch = []
        for rid, tokens, want in entries:
            if not tokens or any(not 0 <= w < len(tokens) for w in want):
                raise ValueError(f"request {rid!r}: an entry needs tokens, and wanted places among them")
            seq = self.live.get(rid)
            if seq is None:
                seq = self.live[rid] = CachedSequence(self.alloc, self.slots, self.engine.max_blocks)
            start, table = seq.extend(len(tokens))
            batch.append(Entry(np.asarray(tokens, dtype=np.int32), start, table, seq.slot, list(want)))
        if not batch:
            return None
        logits = self.engine.step_logits(batch).cpu().numpy()
        self.engine.check_device()
        return logits if logits.shape[0] else None

    def end(self, rid) -> None:
        seq = self.live.pop(rid, None)
        if seq is not None:
            seq.release()


def build_engine(model_dir: str, dtype: str, max_tokens: int, device: str = "cuda:0"):
    """The serving engine of a model directory with a pool of ``max_tokens`` tokens."""
    from ..checkpoint import st
    from ..models.config import HybridConfig, config_from_json
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = config_from_json(json.load(f))
    if isinstance(cfg, HybridConfig):
        from .. import _host
        from ..ops import _cuda
        _host.use_hybrid_library()
        _cuda.use_hybrid_library()
    from .engine import make_engine
    model, _, _ = st.load_model(model_dir)
    tokens = -(-max(max_tokens, 1) // ROUND) * ROUND
    block = 16
    return make_engine(model, block_size=block, num_blocks=tokens // block, max_seq_len=tokens, state_slots=MAX_LIVE,
                       dtype={"bfloat16": "bf16", "float32": "fp32"}[dtype], device=device)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a token trace through a model")
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for the logits of each step")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    a = ap.parse_args(argv)
    session = TraceSession(build_engine(a.model, a.dtype, a.max_tokens))
    os.makedirs(a.out, exist_ok=True)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = session.step([(e["id"], e["tokens"], e.get("want", [])) for e in s["entries"]])
        if logits is not None:
            logits.astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        for rid in s.get("end", []):
            session.end(rid)
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
