"""Replay of a recorded batch schedule: given token ids, step by step, through the engine's page pool and model runner.

A user who wants to see what a model computed in a served mix of requests (portions of prompts beside single decoded tokens, pages
that earlier requests held) feeds the same steps again and reads the logits at chosen places; nothing is sampled.  ``bin/trace_run``
is the command line of it.
"""
from __future__ import annotations

import json
import math
import sys
from pathlib import Path

import torch

from ..ops import _lib
from .engine import LLMEngine
from .runner import EngineConfig

MAX_LIVE = 4                     # requests that hold pages (or state slots) at any time


class _Live:
    def __init__(self, state_slot: int):
        self.pages: list[int] = []
        self.n = 0               # tokens in the cache
        self.state_slot = state_slot


class Replay:
    """Steps over an engine's page manager, state slots and runner; the scheduler's own decisions come from the schedule."""

    def __init__(self, engine: LLMEngine):
        self.eng = engine
        self.live: dict[str, _Live] = {}

    def step(self, entries, end=()):
        """``entries``: (request id, token ids, places whose logits are wanted) of one batch.  Returns fp32 logits
        ``[places, vocab]`` in the order of the entries (None when nothing is wanted) and gives back what ``end`` held."""
        eng, runner = self.eng, self.eng.runner
        batch = []
        for rid, tokens, want in entries:
            if not tokens:
                if want:
                    raise ValueError(f"request {rid}: places wanted of an empty portion")
                continue
            r = self.live.get(rid)
            if r is None:
                if runner.state_slots and not eng.state_free:
                    raise RuntimeError("more live requests than state slots")
                r = self.live[rid] = _Live(eng.state_free.pop() if runner.state_slots else -1)
            need = eng._pages_needed(r.n + len(tokens)) - len(r.pages)
            if need > 0:
                pages = eng.pm.alloc(need)
                if pages is None:
                    raise RuntimeError("the page pool is too small for the live requests")
                r.pages.extend(pages)
            batch.append((r, [int(t) for t in tokens], [int(w) for w in want]))
        logits = None
        if batch and all(len(t) == 1 and r.n > 0 for r, t, _ in batch):
            # one token per request: the decode path (captured graph of the batch-size bucket)
            rows = [i for i, (_, _, w) in enumerate(batch) if w]
            _, out = runner.decode([t[0] for _, t, _ in batch], [r.n for r, _, _ in batch], [r.pages for r, _, _ in batch], want_logits=bool(rows),
                                   state_slots=[r.state_slot for r, _, _ in batch] if runner.state_slots else None)
            if rows:
                logits = torch.cat([out[i:i + 1].expand(len(batch[i][2]), -1) for i in rows])
        elif batch:
            logits = runner.prefill([(t, r.n, r.pages, w, r.state_slot) for r, t, w in batch])
        for r, t, _ in batch:
            r.n += len(t)
        out = logits.float().cpu() if logits is not None else None
        if runner.device.type == "cuda":
            torch.cuda.synchronize()
            _lib.check_device_errors()
        for rid in end:
            self.finish(rid)
        return out

    def finish(self, rid) -> None:
        r = self.live.pop(rid, None)
        if r is None:
            return
        self.eng.pm.release(r.pages)
        if r.state_slot >= 0:
            self.eng.state_free.append(r.state_slot)


def open_engine(model_dir, dtype=torch.bfloat16, max_tokens: int = 8192, device="cuda", max_live: int = MAX_LIVE) -> LLMEngine:
    """An engine whose pool holds ``max_tokens`` tokens of at most ``max_live`` requests (each rounds up to whole pages)."""
    from ..loader.hf import load_model

    cfg = EngineConfig(max_batch=max_live, max_context=max(1, max_tokens), prefix_cache=False, graph_batch_sizes=[1, 2, 4, 8])
    model = load_model(model_dir, device=device, dtype=dtype)
    # a request's count is rounded up to 64 in max_tokens, here to a page: at most (page - 64) more tokens per live request
    pages = math.ceil((max_tokens + max_live * max(0, cfg.page_len - 64)) / cfg.page_len)
    cfg.max_context = pages * cfg.page_len
    return LLMEngine(model, cfg, num_pages=pages, eos_token_ids=[])


def run(lines, engine: LLMEngine, out_dir, emit=print) -> None:
    """``lines``: JSON objects ``{"step", "entries": [{"id", "tokens", "want"}], "end": [...]}``.  Writes ``<step>.f32`` for steps that
    want logits and reports ``done <step>`` after each."""
    rp = Replay(engine)
    out_dir = Path(out_dir)
    for line in lines:
        if not line.strip():
            continue
        st = json.loads(line)
        logits = rp.step([(e["id"], e["tokens"], e.get("want") or []) for e in st["entries"]], st.get("end") or [])
        if logits is not None:
            logits.contiguous().numpy().astype("<f4").tofile(out_dir / f"{st['step']}.f32")
        emit(f"done {st['step']}")
        sys.stdout.flush()


def main(argv=None) -> int:
    import argparse

    ap = argparse.ArgumentParser("trace_run", description="Replay a schedule of token ids read from standard input and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32 (little-endian fp32 [places, vocab])")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at any time")
    ap.add_argument("--device", default="cuda")
    a = ap.parse_args(argv)
    if a.device.startswith("cuda"):
        from ..build import ensure_for

        ensure_for(a.model)
    torch.backends.cuda.matmul.allow_tf32 = False
    eng = open_engine(a.model, getattr(torch, a.dtype), a.max_tokens, a.device)
    run(sys.stdin, eng, a.out, lambda s: print(s, flush=True))
    return 0
