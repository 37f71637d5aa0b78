"""Replays given token ids through a served model, step by step, and writes the logits that each step asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Every input line is one step, a JSON object: {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}],
"end": []}.  `tokens` are a request's next tokens, `want` the places among them whose logits are written, `end` the
requests whose pages and state slot are given back after the step; at most four are live at any time.  All entries of a step are one batch of `ModelRunner.step`, the call
the serving engine makes: portions of prompts beside single decoded tokens, steps of decoded tokens alone from a CUDA
graph.  A step with wanted places writes OUT/<step>.f32 (little-endian 32-bit floats [wanted, vocab], in the order of the
entries and of `want`); after every step a line "done <step>" is printed.  Nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 16
LIVE_REQUESTS = 4                     # state slots of models with recurrent layers


def parse_args(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="replay token ids through a served model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="most tokens that live requests hold at any time; the KV cache is made for this many")
    ap.add_argument("--device", default="cuda:0")
    return ap.parse_args(argv)


class TraceReplay:
    """Admits requests at their first entry, grows their pages with every entry, and frees them when they end."""

    def __init__(self, runner):
        self.runner = runner
        self._seq: dict = {}              # request id -> (sequence id of the cache, tokens so far)
        self._next = 0

    def _grow(self, rid: str, n: int) -> tuple:
        seq, have = self._seq.get(rid, (None, 0))
        if seq is None:
            seq, self._next = self._next, self._next + 1
        if not self.runner.cache.allocate(seq, have + n):
            raise RuntimeError(f"request {rid!r} does not fit in the cache")
        self._seq[rid] = (seq, have + n)
        return seq, have

    def step(self, entries: list, end: list):
        """Runs one step; returns the wanted logits [wanted, vocab] as an fp32 CPU tensor, or None."""
        import torch
        chunks, chunk_of, dec, dec_of = [], {}, [], {}
        for i, e in enumerate(entries):
            toks = e["tokens"]
            if not toks:
                continue
            seq, have = self._grow(e["id"], len(toks))
            if len(toks) == 1 and have > 0:
                dec_of[i] = len(dec)
                dec.append((seq, toks[0], have + 1))
            else:
                chunk_of[i] = len(chunks)
                chunks.append((seq, toks, have, list(e["want"])))
        got, dec_logits = self.runner.step(chunks, [d[0] for d in dec], [d[1] for d in dec], [d[2] for d in dec])
        vocab = self.runner.cfg.vocab_size
        parts = []
        for i, e in enumerate(entries):
            if not e["want"]:
                continue
            lg = got[chunk_of[i]] if i in chunk_of else dec_logits[dec_of[i]:dec_of[i] + 1].expand(len(e["want"]), -1)
            parts.append(lg[:, :vocab].float().cpu())
        for rid in end:
            self.runner.cache.free(self._seq.pop(rid)[0])
        return torch.cat(parts) if parts else None


def main(argv=None) -> int:
    a = parse_args(argv)
    from ..models.registry import architecture, ensure_kernels, load_config
    cfg = load_config(a.model)
    if a.dtype == "float32" and not a.device.startswith("cpu") and not architecture(cfg.arch).float32:
        print(f"{cfg.arch} does not run in 32-bit on a GPU", file=sys.stderr)
        return 3
    if not a.device.startswith("cpu"):
        ensure_kernels(cfg.arch)
    import torch

    from .model_runner import load_runner
    if not a.device.startswith("cpu"):
        if not torch.cuda.is_available():
            raise RuntimeError("trace_run needs a CUDA device")
        torch.cuda.set_device(torch.device(a.device))
    runner = load_runner(a.model, device=a.device, dtype=getattr(torch, a.dtype), num_blocks=max(1, -(-a.max_tokens // PAGE)),
                         block_size=PAGE, num_slots=LIVE_REQUESTS)
    replay = TraceReplay(runner)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        out = replay.step(s["entries"], s["end"])
        if out is not None:
            out.contiguous().numpy().astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        if runner.device.type == "cuda":
            from .. import _native
            _native.raise_on_status()
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
