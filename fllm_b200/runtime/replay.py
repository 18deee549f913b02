"""Replay of a recorded serving trace: given token ids are fed step by step through the engine's own batch building, paged
cache, state rows and forward (captured graphs for pure decode steps), and the logits of chosen tokens are read back.
Nothing is sampled.

A step is ``{"step": n, "entries": [{"id": ..., "tokens": [...], "want": [places among these tokens]}], "end": [ids]}``. A
request is admitted at its first entry, may pause for any number of steps, and gives its blocks and state row back when
it is listed in ``end``.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, Sequence

import torch

from .request import Request, RequestStatus, SamplingParams
from .scheduler import ScheduledSeq, ScheduledStep


class TraceReplay:
    def __init__(self, engine):
        self.eng = engine
        self.live: Dict[str, Request] = {}

    def step(self, entries: Sequence[dict], end: Sequence[str] = ()) -> torch.Tensor:
        """Runs one step; fp32 logits [wanted tokens, vocab] in the order of the entries and their ``want`` lists."""
        eng = self.eng
        step = ScheduledStep()
        for e in entries:
            toks = [int(t) for t in e["tokens"]]
            want = [int(i) for i in e.get("want") or ()]
            if not toks:
                raise ValueError(f"request {e['id']!r}: an entry without tokens")
            if any(not 0 <= t < eng.model_cfg.vocab_size for t in toks) or any(not 0 <= i < len(toks) for i in want):
                raise ValueError(f"request {e['id']!r}: a token id or a wanted place is out of range")
            r = self.live.get(e["id"])
            if r is None:
                r = Request(str(e["id"]), next(eng._seq_ids), toks, SamplingParams(max_tokens=1))
                r.status = RequestStatus.RUNNING
                eng.blocks.allocate(r.seq_id, [])
                self.live[e["id"]] = r
            else:
                r.output.extend(toks)
            if r.num_tokens > eng.cfg.max_model_len or not eng.blocks.ensure_capacity(r.seq_id, r.num_tokens):
                raise RuntimeError(f"request {e['id']!r}: the cache pool has no room for {r.num_tokens} tokens")
            rows = sorted(set(want))                # computed once each, in token order
            step.seqs.append(ScheduledSeq(r, r.num_computed, len(toks), bool(rows), rows=rows))
        logits = eng.run_forced(step)
        out, base = [], 0
        for e, s in zip(entries, step.seqs):
            at = {place: base + k for k, place in enumerate(s.rows)}
            out.extend(at[int(i)] for i in e.get("want") or ())
            base += len(s.rows)
            s.req.num_computed += s.count
            eng.blocks.commit_tokens(s.req.seq_id, s.req.all_tokens, s.req.num_computed)
        for rid in end:
            eng.blocks.free_seq(self.live.pop(rid).seq_id)
        return logits[out]


def make_engine(model: str, dtype: str, max_tokens: int, device: str = "cuda"):
    """An engine whose cache pool holds ``max_tokens`` tokens and whose state pools hold four requests."""
    from ..config import EngineConfig
    from ..formats.loader import load_model
    from .engine import LLMEngine
    f32 = dtype == "float32"
    cfg, weights, _ = load_model(model, device, dtype=torch.float32 if f32 else torch.bfloat16)
    bs = EngineConfig.block_size
    ec = EngineConfig(dtype="fp32" if f32 else "bf16", max_num_seqs=4, spare_state_rows=0, block_size=bs, num_kv_blocks=-(-max_tokens // bs),
                      max_model_len=max_tokens, max_num_batched_tokens=max_tokens, enable_prefix_caching=False)
    return LLMEngine(cfg, ec, device=device, weights=weights)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Feed recorded token ids through a model step by step and write logits.")
    ap.add_argument("--model", required=True, help="directory with config.json and safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for <step>.f32: little-endian fp32 logits [wanted, vocab]")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache pool holds")
    args = ap.parse_args(argv)
    if args.dtype == "float32":
        from ..config import ModelConfig
        with open(os.path.join(args.model, "config.json")) as f:
            if not ModelConfig.from_hf_config(json.load(f)).native_f32:
                print("the kernels of this family run in bf16 only", file=sys.stderr)
                return 3
    if not torch.cuda.is_available():
        print("a CUDA device is needed", file=sys.stderr)
        return 2
    replay = TraceReplay(make_engine(args.model, args.dtype, args.max_tokens))
    for line in sys.stdin:
        if not line.strip():
            continue
        d = json.loads(line)
        logits = replay.step(d["entries"], d.get("end") or ())
        if logits.shape[0]:
            part = os.path.join(args.out, f".{d['step']}.part")
            logits.cpu().numpy().astype("<f4").tofile(part)
            os.replace(part, os.path.join(args.out, f"{d['step']}.f32"))
        code = replay.eng.ops.check_status()
        if code:
            raise RuntimeError(f"kernel status word = {code}")
        print(f"done {d['step']}", flush=True)
    replay.eng.close()
    return 0
