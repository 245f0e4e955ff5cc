"""Replay of a request trace: given token ids go through a model step by step, and chosen logits are written out.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Every input line is one step, ``{"step": n, "entries": [{"id": "a", "tokens": [..], "want": [..]}, ..], "end": ["a", ..]}``:
all entries run as one batch through ``Generator.step`` (portions of prompts beside single tokens, captured decode graphs
when every entry brings one token); a request is admitted at its first entry and gives back its pages and state slot when
it is listed in ``end``. ``want`` lists places among an entry's tokens; their logits go to ``DIR/<step>.f32`` as
little-endian fp32 rows in the order of the entries. ``done <step>`` is printed after every step. The page pool holds
``--max-tokens`` tokens (each live request rounded up to whole pages), the state pool ``--max-seqs`` requests."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Optional


class TraceReplay:
    """The live requests of a trace on one generator."""

    def __init__(self, model, max_tokens: int, max_seqs: int = 4):
        from ..models.generation import Generator
        from ..models.kv_cache import BLOCK
        blocks = -(-max_tokens // BLOCK)
        kw = {"max_seqs": max_seqs} if getattr(model, "slotted_cache", False) else {}
        cache = model.new_cache(blocks, **kw)
        if cache.scratch_block is None:           # captured steps of this cache take their scratch block from the pool
            cache = model.new_cache(blocks + 1, **kw)
        self.gen = Generator(model, cache=cache)
        self.seqs: Dict[str, int] = {}

    def step(self, entries: List[dict], end: List[str]):
        """Logits [wanted, vocab] of one step (fp32 on the host), or None when nothing is wanted."""
        logits = None
        if entries:
            for e in entries:
                if e["id"] not in self.seqs:
                    self.seqs[e["id"]] = self.gen.new_seq()
            out = self.gen.step([self.seqs[e["id"]] for e in entries], [e["tokens"] for e in entries],
                                [e.get("want") or [] for e in entries])
            if out.shape[0]:
                logits = out.float().cpu()
        for rid in end:
            self.gen.cache.free_sequence(self.seqs.pop(rid))
        return logits


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a request trace and write logits")
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="directory for <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-seqs", type=int, default=4, help="most live requests at any time")
    a = ap.parse_args(argv)
    import torch

    from ..models.architectures import PAGED_FAMILIES, family_of
    from ..models.loader import load_pretrained
    from ..ops import native
    with open(os.path.join(a.model, "config.json"), "r", encoding="utf-8") as fh:
        config = json.load(fh)
    fam = family_of(config)
    if fam not in PAGED_FAMILIES:
        print(f"error: {fam or 'unknown'} models are not served from the paged caches", file=sys.stderr)
        return 2
    native.require(str(config.get("architecture", config.get("model_type"))).lower() if fam == "hybrid" else "decoder")
    if not native.available():
        print(f"error: no CUDA device or native library ({native.load_error()})", file=sys.stderr)
        return 2
    torch.backends.cuda.matmul.allow_tf32 = False
    model, _, _ = load_pretrained(a.model, getattr(torch, a.dtype), "cuda")
    model.eval()
    for p in model.parameters():
        p.requires_grad_(False)
    os.makedirs(a.out, exist_ok=True)
    replay = TraceReplay(model, a.max_tokens, a.max_seqs)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step["entries"], step.get("end") or [])
        if logits is not None:
            part = os.path.join(a.out, f".{step['step']}.part")
            logits.numpy().astype("<f4").tofile(part)
            os.replace(part, os.path.join(a.out, f"{step['step']}.f32"))
        else:
            torch.cuda.synchronize()
        print(f"done {step['step']}", flush=True)
    native.check_status()
    return 0


if __name__ == "__main__":
    sys.exit(main())
