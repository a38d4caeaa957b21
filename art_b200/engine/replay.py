"""Feeds given token ids through an engine's runner step by step and reports logits: nothing is sampled.

A trace is a stream of steps; each brings the next tokens of some requests (portions of prompts beside single tokens) and
names the places whose logits are wanted.  Every step is one batch of the runner (``DeviceRunner.step_logits``), on the
block manager, cache and state slots the engine generates with.  Requests are admitted at their first entry, may be left
out of steps, and give everything back when they end.

``bin/trace_run`` is this module's command line::

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N [--slots S]  < steps.jsonl

reading ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}`` lines; logits go to ``OUT/<n>.f32``
(little-endian fp32, wanted rows x vocabulary), ``done <n>`` to standard output.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from dataclasses import dataclass, field

import torch

from .kv_cache import BlockManager
from .runner import SeqView

BLOCK_SIZE = 16
UNSUPPORTED_DTYPE_EXIT = 3


@dataclass
class _Request:
    tokens: list[int] = field(default_factory=list)
    blocks: list[int] = field(default_factory=list)
    state_slot: int = -1


class Replay:
    def __init__(self, runner, bm: BlockManager, kv):
        self.runner, self.bm = runner, bm
        self.state_slots = getattr(kv, "state_slots", None)
        self.live: dict[str, _Request] = {}

    def step(self, entries: list[dict], end: list[str] = ()) -> torch.Tensor:
        """fp32 logits ``[wanted, vocab]`` in the order of the entries and of their ``want`` lists."""
        bs, vocab = self.bm.block_size, self.runner.cfg.vocab_size
        views, want = [], []
        for e in entries:
            new = e["tokens"]
            if not new or min(new) < 0 or max(new) >= vocab:
                raise ValueError(f"request {e['id']}: tokens must be a non-empty list of ids below {vocab}")
            if any(not 0 <= w < len(new) for w in e.get("want", [])):
                raise ValueError(f"request {e['id']}: wanted places lie outside its new tokens")
            r = self.live.get(e["id"])
            if r is None:
                r = self.live[e["id"]] = _Request()
                if self.state_slots is not None:
                    slot = self.state_slots.alloc()
                    if slot is None:
                        raise RuntimeError("no state slot is free")
                    r.state_slot = slot
            n0 = len(r.tokens)
            r.tokens += new
            need = (len(r.tokens) + bs - 1) // bs - len(r.blocks)
            fresh = self.bm.alloc(need)
            if fresh is None:
                raise RuntimeError("no cache block is free")
            r.blocks += fresh
            views.append(SeqView(r.tokens, n0, r.blocks, -1, 0.0, 0, 0, state_slot=r.state_slot))
            want.append(e.get("want", []))
        logits = (self.runner.step_logits(views, want) if views
                  else torch.empty((0, vocab), dtype=torch.float32, device=self.runner.device))
        for i in end:
            r = self.live.pop(i)
            self.bm.free(r.blocks)
            if r.state_slot >= 0:
                self.state_slots.free(r.state_slot)
        return logits


def main(argv: list[str] | None = None) -> int:
    from ..models.config import ModelConfig
    from ..models.hybrid import HybridConfig
    from ..models.weights import load_base_weights
    from ..ops import _lib
    from .factory import UnsupportedPrecision, build_runner

    ap = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits files")
    ap.add_argument("--max-tokens", type=int, required=True, help="size of the cache pool in tokens")
    ap.add_argument("--slots", type=int, default=4, help="live requests (state slots)")
    a = ap.parse_args(argv)
    cfg = ModelConfig.from_pretrained_dir(a.model)
    if isinstance(cfg, HybridConfig):
        from .hybrid_runner import kernel_sources

        _lib.require(kernel_sources(cfg))
    blocks = (a.max_tokens + BLOCK_SIZE - 1) // BLOCK_SIZE
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    base = load_base_weights(a.model, cfg, device=dev)
    try:
        runner, kv = build_runner(cfg, base, num_blocks=blocks, block_size=BLOCK_SIZE, num_slots=a.slots, device=dev,
                                  dtype=getattr(torch, a.dtype), max_loras=1)
    except UnsupportedPrecision as e:
        print(e, file=sys.stderr)
        return UNSUPPORTED_DTYPE_EXIT
    rep = Replay(runner, BlockManager(blocks, BLOCK_SIZE, False), kv)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = rep.step(s["entries"], s.get("end", []))
        if logits.shape[0]:
            data = logits.contiguous().cpu().numpy().astype("<f4").tobytes()
            with open(os.path.join(a.out, f"{s['step']}.f32"), "wb") as f:
                f.write(data)
        _lib.check_status(dev)
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
