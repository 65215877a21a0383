"""Command-line programs over model folders: bin/trace_run and bin/generate."""
from __future__ import annotations

import argparse
import json
import os
import sys


def _torch_cuda():
    import torch
    if not torch.cuda.is_available():
        raise SystemExit("no CUDA device (there is no CPU fallback)")
    torch.cuda.set_device(0)
    return torch


def _check_status(stack) -> None:
    code = stack.device_status()
    if code:
        raise RuntimeError(f"device status {code}: a kernel gave up or refused its input")


class TraceRunner:
    """Feeds given tokens through a stack's continuous-batching rows and returns logits; samples nothing."""

    def __init__(self, torch, stack):
        self.torch, self.stack = torch, stack
        self.ids: list[str] = []           # ids[r] = request in row r
        stack.begin_batching()

    def run(self, entries: list[dict]):
        rows = []
        for e in entries:
            if e["id"] not in self.ids:
                self.stack.open()
                self.ids.append(e["id"])
            if not e["tokens"]:
                continue
            toks = self.torch.tensor(e["tokens"], dtype=self.torch.int32, device="cuda")
            want = sorted(set(e.get("want") or []))
            logits = self.stack.extend(self.ids.index(e["id"]), toks, want)
            rows += [logits[want.index(w)] for w in (e.get("want") or [])]
        return self.torch.stack(rows).cpu().numpy() if rows else None

    def end(self, request: str) -> None:
        if request not in self.ids:
            return
        row = self.ids.index(request)
        self.stack.retire(row)             # the last row moves into the freed place
        last = self.ids.pop()
        if row < len(self.ids):
            self.ids[row] = last


def trace_main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replays steps of token ids read from standard input and writes the wanted logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=8, help="most live requests")
    a = ap.parse_args(argv)
    from . import build, models
    build.build_library()
    torch = _torch_cuda()
    pages = -(-a.max_tokens // 64) + 2 * a.max_requests        # every live request may leave its last page part-filled
    stack = models.load_model(a.model, models.Limits(a.max_requests, a.max_tokens, pages, min(max(a.max_tokens, a.max_requests), 8192), a.dtype))
    with torch.cuda.stream(torch.cuda.Stream()):
        runner = TraceRunner(torch, stack)
        for line in sys.stdin:
            if not line.strip():
                continue
            step = json.loads(line)
            logits = runner.run(step.get("entries", []))
            for request in step.get("end", []):
                runner.end(request)
            _check_status(stack)
            if logits is not None:
                logits.astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
            print(f"done {step['step']}", flush=True)
    return 0


def generate_main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="generate", description="Greedy generation for prompts of token ids, one JSON list per line of standard input.")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--eos", type=int, default=None)
    ap.add_argument("--max-seqs", type=int, default=8, help="sequences in flight")
    ap.add_argument("--max-seq-len", type=int, default=4096)
    a = ap.parse_args(argv)
    from . import batching, build, models
    build.build_library()
    torch = _torch_cuda()
    stack = models.load_model(a.model, models.Limits(a.max_seqs, a.max_seq_len, 0, 0, a.dtype))
    prompts = [json.loads(line) for line in sys.stdin if line.strip()]
    with torch.cuda.stream(torch.cuda.Stream()):
        done = batching.generate(stack, prompts, a.max_new_tokens, a.eos)
        _check_status(stack)
    for tokens in done:
        print(json.dumps(tokens))
    return 0
