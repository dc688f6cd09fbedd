"""Replay of a recorded schedule: token ids arrive step by step for named requests, and logits are read at chosen places.

Nothing is sampled and nothing is decided here: every step is one batch through the engine's scheduler bookkeeping, block
manager and model runner, the same step function that generation uses (captured decode graphs included).  A line of a
trace is a JSON object

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

`main` is the command-line form (bin/trace_run): it writes the wanted logits of a step to DIR/<step>.f32 (little-endian
fp32, [wanted, vocab], in the order of the entries) and answers each line with "done <step>".
"""
from __future__ import annotations

import argparse
import json
import os
import sys

from .llm_engine import LLMEngine
from .sequence import Sequence, SequenceStatus


class ReplaySession:
    def __init__(self, engine: LLMEngine):
        self.engine = engine
        self.live: dict = {}

    def _feed(self, rid, tokens: list) -> Sequence:
        vocab, limit = self.engine.config.model_config.vocab_size, self.engine.config.max_model_len
        if not tokens or any(not 0 <= t < vocab for t in tokens):
            raise ValueError(f"request {rid!r}: tokens must be ids in [0, {vocab})")
        seq = self.live.get(rid)
        if seq is None:
            seq = self.live[rid] = Sequence(tokens)
        else:
            seq.extend(tokens)
        if seq.num_tokens > limit:
            raise ValueError(f"request {rid!r} has {seq.num_tokens} tokens, the model takes {limit}")
        self.engine.scheduler.schedule_given(seq)
        return seq

    def step(self, entries: list, end=()):
        """Runs one batch; returns fp32 logits [wanted, vocab] on the host, or None when nothing is wanted."""
        seqs, rows, base = [], [], 0
        for e in entries:
            tokens = [int(t) for t in e["tokens"]]
            seqs.append(self._feed(e["id"], tokens))
            rows += [base + int(k) for k in e.get("want", ())]
            base += len(tokens)
        logits = self.engine.model_runner.run_logits(seqs, rows) if seqs else None
        for seq in seqs:
            self.engine.scheduler.finish_given(seq)
        for rid in end:
            self.close(rid)
        return logits if rows else None

    def close(self, rid):
        """Gives back the blocks and the state slot of a request."""
        seq = self.live.pop(rid, None)
        if seq is not None:
            self.engine.scheduler.running.pop(seq.seq_id, None)
            self.engine.scheduler.deallocate(seq)
            self.engine.model_runner.free_deltanet_slot(seq.seq_id)
            seq.status = SequenceStatus.FINISHED


def make_engine(model: str, dtype: str, max_tokens: int, device: str = "cuda", max_live: int = 4) -> LLMEngine:
    """An engine whose cache holds `max_tokens` tokens (each request rounded up to a whole block) and `max_live` requests."""
    blocks = max(1, -(-max_tokens // 16))
    return LLMEngine(model, quantization={"bfloat16": "bf16", "float32": "fp32"}[dtype], device=device, tokenizer="ids",
                     num_kvcache_blocks=blocks, max_num_seqs=max_live, max_model_len=16 * blocks,
                     max_num_batched_tokens=max(16, max_tokens), enable_prefix_caching=False)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description="replay a schedule of token ids and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at most")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"])
    args = ap.parse_args(argv)
    os.makedirs(args.out, exist_ok=True)
    try:
        engine = make_engine(args.model, args.dtype, args.max_tokens, args.device)
    except ValueError as e:
        if args.dtype == "float32" and "quantization" in str(e):
            print(f"no 32-bit mode: {e}", file=sys.stderr)
            return 3
        raise
    session = ReplaySession(engine)
    for line in sys.stdin:
        if not line.strip():
            continue
        req = json.loads(line)
        logits = session.step(req["entries"], req.get("end", ()))
        if logits is not None:
            logits.contiguous().numpy().astype("<f4", copy=False).tofile(os.path.join(args.out, f"{req['step']}.f32"))
        print(f"done {req['step']}", flush=True)
    engine.close()
    return 0
