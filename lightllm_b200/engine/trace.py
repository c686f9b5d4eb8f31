"""Replays given token ids through a model, step by step, and reports logits (`bin/trace_run`).

The engine is the offline `LLM`: its model, KV pool, request table, weight loading and kernels.  Every step of the
trace is one `ModelBackend.replay_step`: the tokens it brings run on top of what earlier steps left in the pool, a decode
step when each request brings one token, else one prompt pass with portions of prompts beside single tokens.  Nothing is
sampled, and no prefix is shared between requests.

Input, one JSON object per line:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}
Output: DIR/<step>.f32 with the logits at the wanted places (little-endian fp32, [wanted, vocab], in the order of the
entries), and the line "done <step>" after every step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

MAX_LIVE = 4      # requests that are live at any time
EXIT_NO_FP32 = 3


class TraceReplayer:
    def __init__(self, llm):
        self.llm = llm
        self.backend = llm.backend
        self.live = {}

    @classmethod
    def open(cls, model_dir: str, dtype: str, max_tokens: int, max_live: int = MAX_LIVE, **kw):
        from .llm import LLM

        llm = LLM(model_dir=model_dir, data_type=dtype, max_total_token_num=max_tokens, running_max_req_size=max_live,
                  max_req_total_len=max_tokens, disable_dynamic_prompt_cache=True, **kw)
        return cls(llm)

    def _admit(self, name, tokens):
        limit = self.llm.args.max_req_total_len
        req = self.llm._new_req(list(tokens), {"max_new_tokens": max(limit - len(tokens), 1)})
        self.live[name] = self.backend.add_reqs([req])[0]

    def step(self, entries, end=()):
        """entries: [(name, new tokens, wanted places among them)] -> fp32 logits [wanted, vocab] on the host."""
        items, rows, base = [], [], 0
        for name, tokens, want in entries:
            if name in self.live:
                for t in tokens:
                    self.live[name].append_token(int(t), 0.0)
            else:
                self._admit(name, tokens)
            items.append((self.live[name], len(tokens)))
            rows += [base + int(w) for w in want]
            base += len(tokens)
        logits = self.backend.replay_step(items, rows).float().cpu().numpy() if items else None
        for name in end:
            ir = self.live.pop(name)
            self.backend.ctx.remove_req(ir)
            ir.shm_req.release_shm_arrays()
        return logits


def parse_args(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="feed given token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="size of the KV pool in tokens")
    ap.add_argument("--device", choices=("cuda", "cpu"), default="cuda",
                    help="cpu: the plain PyTorch restatements of the operators (for tests)")
    return ap.parse_args(argv)


def main(argv=None) -> int:
    a = parse_args(argv)
    from ..models.base import load_config
    from ..models.registry import get_model_class
    from ..ops import _native
    from ..parallel import dist as pdist

    if a.device == "cuda" and not torch.cuda.is_available():
        print("trace_run: no CUDA device", file=sys.stderr)
        return 1
    cls = get_model_class(load_config(a.model))
    if a.dtype == "float32" and a.device == "cuda" and not cls.supports_float32:
        print(f"trace_run: {cls.__name__} has no float32 path on the GPU", file=sys.stderr)
        return EXIT_NO_FP32
    if a.device == "cuda":
        _native.prepare(cls.native_units)
        torch.cuda.set_device(0)
    ps = pdist.ParallelState(device=torch.device("cuda", 0) if a.device == "cuda" else torch.device("cpu"))
    rep = TraceReplayer.open(a.model, a.dtype, a.max_tokens, pstate=ps)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        entries = [(e["id"], e["tokens"], e.get("want", ())) for e in s.get("entries", ()) if e["tokens"]]
        logits = rep.step(entries, s.get("end", ()))
        if any(len(w) for _, _, w in entries):
            logits.astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    rep.llm.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
