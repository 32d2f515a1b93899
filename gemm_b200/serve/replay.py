"""Replay of a trace of engine steps: given token ids go through the engine in the given portions, and logits come out; nothing is
sampled and nothing is scheduled.

``Replay`` drives what the serving loop drives: the block manager and the state slots of an ``LLM``, its batch assembly
(``LLM.build_batch``) and the model's step.  A request is admitted at its first entry and keeps its pages and slot until it is ended;
it may be left out of steps in between.

``python -m gemm_b200.serve.replay`` (``bin/trace_run``) reads steps as JSON lines from standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

writes the wanted logits of each step to ``<out>/<step>.f32`` (little-endian f32, [wanted, vocab], in the order of the entries), and
prints ``done <step>`` after every step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from dataclasses import dataclass
from typing import Dict, Iterable, Optional, Sequence

import torch

from .llm import LLM

FORMATS = {"bfloat16": "bf16", "float32": "f32"}
PAGE = 64
MAX_LIVE = 4


@dataclass
class _Live:
    seq: int
    slot: int
    length: int = 0


class Replay:
    def __init__(self, llm: LLM):
        self.llm = llm
        self.live: Dict[str, _Live] = {}

    @torch.no_grad()
    def step(self, entries: Sequence[dict], end: Iterable[str] = ()) -> Optional[torch.Tensor]:
        """Run one step; returns the wanted logits f32 ``[wanted, vocab]`` on the host (None if none are wanted)."""
        llm = self.llm
        seqs, slots, q_lens, ctx, ids, rows = [], [], [], [], [], []
        seen = set()
        for e in entries:
            toks, rid = e["tokens"], e["id"]
            if rid in seen:
                raise ValueError(f"request {rid!r} appears twice in one step")
            seen.add(rid)
            if not toks:
                continue
            if any(not 0 <= t < llm.cfg.vocab for t in toks):
                raise ValueError(f"request {rid!r}: token id outside the vocabulary")
            r = self.live.get(rid)
            if r is None:
                if not llm._free_slots:
                    raise MemoryError("no state slot is free")
                r = self.live[rid] = _Live(llm.blocks.new_sequence(), llm._free_slots.pop())
            llm.blocks.reserve(r.seq, r.length + len(toks))
            rows.extend(len(ids) + w for w in e.get("want", ()))
            seqs.append(r.seq); slots.append(r.slot); q_lens.append(len(toks)); ctx.append(r.length)
            ids.extend(toks)
            r.length += len(toks)
        out = None
        if seqs:
            fb = llm.build_batch(seqs, slots, q_lens, ctx, ids, rows)
            if rows:
                out = llm.model.forward(fb).float().cpu()
            else:
                llm.model.forward_hidden(fb)
        for rid in end:
            r = self.live.pop(rid, None)
            if r is not None:
                llm.blocks.release(r.seq)
                llm._free_slots.append(r.slot)
        return out


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of engine steps and write logits")
    ap.add_argument("--model", required=True, help="checkpoint directory (config.json + *.safetensors)")
    ap.add_argument("--dtype", default="bfloat16", choices=sorted(FORMATS), help="bfloat16: as served; float32: every product and activation in 32-bit")
    ap.add_argument("--out", required=True, help="directory for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at any time (each rounded up to whole pages)")
    args = ap.parse_args(argv)
    from .. import _native
    from ..models import loader
    from ..models.config import LAYERED_ARCHS
    if not torch.cuda.is_available():
        sys.exit("trace_run needs a CUDA device")
    with open(os.path.join(args.model, "config.json")) as fh:
        layered = json.load(fh).get("architecture") in LAYERED_ARCHS
    if not layered and args.dtype == "float32":
        print("32-bit inference is built for models described layer by layer only", file=sys.stderr)
        return 3
    if layered:
        _native.use_subset("layered")          # compile no more than this model family needs
    llm = LLM(loader.load_safetensors(args.model, FORMATS[args.dtype], "cuda"), None, max_running=MAX_LIVE, num_pages=max(1, (args.max_tokens + PAGE - 1) // PAGE),
              page_size=PAGE)
    rep = Replay(llm)
    for line in sys.stdin:
        if not line.strip():
            continue
        st = json.loads(line)
        logits = rep.step(st["entries"], st.get("end", ()))
        if logits is not None:
            with open(os.path.join(args.out, f"{st['step']}.f32"), "wb") as fh:
                fh.write(logits.contiguous().numpy().astype("<f4").tobytes())
        _native.assert_status_ok()
        print(f"done {st['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
