"""Trace replay: feeds given token ids through the serving engine's own step functions and writes the logits it asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps are read from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step are one batch.  A single token of a request that is already running is a decode row, everything else a ragged
prefill item (a prompt or a portion of one), so a step is what the scheduler would launch: a decode graph, a prefill, or one mixed
pass over both.  For a step that wants logits, DIR/<step>.f32 holds them, [wanted, vocab] little-endian fp32, in the order of the
entries and of `want`; `done <step>` follows on standard output.
"""

from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List

import torch

from ..config import EngineConfig, ModelConfig
from ..models.decoder import DecoderModel
from ..utils.weights import Weights, weight_files
from .kv_cache import BlockAllocator, make_cache
from .runner import ModelRunner, PrefillItem

MAX_REQUESTS = 4


class TraceReplay:
    """Requests by name over one cache pool of `max_tokens` tokens and a few state slots."""

    def __init__(self, model: DecoderModel, max_tokens: int, max_requests: int = MAX_REQUESTS, page: int = 32):
        self.model = model
        blocks = (max_tokens + page - 1) // page + 1            # block 0 belongs to no request
        self.kv = make_cache(model, EngineConfig(), blocks, max_requests, page, num_slots=max_requests + 1)
        self.alloc = BlockAllocator(blocks, page, model.config.sliding_window)
        self.runner = ModelRunner(model, self.kv, max_batch=max_requests, max_seq_tokens=max_tokens, max_prefill_tokens=max(max_tokens, 64))
        self.runner.keep_logits = True
        self.held: Dict[str, List[int]] = {}
        self.length: Dict[str, int] = {}

    def _slot(self, rid: str) -> int:
        slots = self.kv.state_slots
        if slots is None:
            return 0
        slot = slots.acquire(rid)
        if slot is None:
            raise RuntimeError("more requests are live than there are state slots")
        return slot

    def step(self, entries: List[dict]) -> torch.Tensor:
        """Runs the entries as one batch -> logits [wanted, vocab] fp32 on the host."""
        run = self.runner
        dec, items, rows_of = [], [], []
        for e in entries:
            rid, toks = e["id"], e["tokens"]
            blocks = self.held.setdefault(rid, [])
            before = self.length.get(rid, 0)
            if not self.alloc.extend(blocks, before + len(toks)):
                raise RuntimeError("the cache pool is full")
            slot = self._slot(rid)
            self.length[rid] = before + len(toks)
            if len(toks) == 1 and before > 0:
                rows_of.append(("d", len(dec)))
                dec.append((toks[0], before, list(blocks), slot))
            else:
                rows_of.append(("p", sum(len(it.logit_rows) for it in items)))
                items.append(PrefillItem(toks, before, list(blocks), state_slot=slot, logit_rows=list(e["want"])))
        if dec:
            rows = [run.state.take_row(i) for i in range(len(dec))]
            run.install(rows, [d[0] for d in dec], [d[1] for d in dec], [d[2] for d in dec], [0] * len(dec), [d[3] for d in dec])
            run.resort()
        if dec and items:
            run.mixed_step(items)
            logits = run.last_logits
        elif dec:
            _, _, logits = run.decode(need_logits=True)
        else:
            _, _, logits = run.prefill(items)
        want = []
        for e, (kind, at) in zip(entries, rows_of):
            base = at if kind == "d" else (len(dec) + at)
            want += [base + (0 if kind == "d" else i) for i in range(len(e["want"]))]
        out = logits.index_select(0, torch.tensor(want, device=logits.device)).float().cpu() if want else torch.empty(0, self.model.vocab)
        if dec:
            run.retire(list(range(len(dec))))
            for r in list(run.state.live):
                run.state.drop_row(r)
            run.resort()
        if self.model.device.type == "cuda":
            from ..ops import native
            native.workspace(self.model.device).check_status()
        return out

    def end(self, rid: str):
        self.alloc.release(self.held.pop(rid, []))
        self.length.pop(rid, None)
        if self.kv.state_slots is not None:
            self.kv.state_slots.release(rid)


def load_model(path: str, dtype: torch.dtype, device, max_positions: int) -> DecoderModel:
    config = ModelConfig.from_pretrained(path)
    return DecoderModel.from_weights(config, Weights(weight_files(path), device="cpu", dtype=dtype), device, dtype, max_positions=max_positions)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of given tokens through a model and write its logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder that takes <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens the live requests hold at any time")
    ap.add_argument("--device", default="cuda", help="cuda, or cpu for the plain PyTorch operators")
    args = ap.parse_args(argv)
    dtype = getattr(torch, args.dtype)
    config = ModelConfig.from_pretrained(args.model)
    if args.device != "cpu" and dtype == torch.float32 and config.layer_specs is None:
        print(f"{config.model_type} has no 32-bit kernels", file=sys.stderr)
        return 3
    if args.device != "cpu":
        from ..ops import native
        if config.layer_specs is not None:
            native.use_subset("mixers")
        native.load()
    with torch.inference_mode():
        model = load_model(args.model, dtype, args.device, args.max_tokens + 64)
        replay = TraceReplay(model, args.max_tokens)
        for line in sys.stdin:
            if not line.strip():
                continue
            s = json.loads(line)
            logits = replay.step(s["entries"]) if s["entries"] else torch.empty(0, model.vocab)
            if logits.shape[0]:
                path = os.path.join(args.out, f"{s['step']}.f32")
                logits.numpy().astype("<f4").tofile(path)
            for rid in s.get("end", []):
                replay.end(rid)
            print(f"done {s['step']}", flush=True)
    return 0
