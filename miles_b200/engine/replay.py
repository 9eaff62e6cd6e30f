"""Replay of recorded token streams through an engine, with the logits they produce.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come on standard input, one JSON object a line:
``{"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}``. Every entry's tokens continue
its sequence (``Engine.feed``: the model, cache manager and kernels that generation uses, nothing is sampled); ``want``
names places among them whose logits are wanted, ``end`` the sequences that are finished after the step. A step with wanted
logits writes ``<out>/<step>.f32`` (little-endian fp32, ``[wanted, vocab]``, entries in order); every step prints
``done <step>``.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def build_engine(model_dir: str, dtype: str, max_tokens: int, device: str = "cuda", page_size: int = 64, max_running: int = 64):
    """The engine that serves a checkpoint directory in ``dtype``, its cache sized for ``max_tokens`` live tokens."""
    import torch

    from ..checkpoint import load_hf
    from ..models import ParamStore, build_model, get_config
    from .core import Engine

    # "float32" means 32-bit products, not a reduced-precision matrix mode
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cudnn.allow_tf32 = False
    cfg = get_config(model_dir)
    store = ParamStore(cfg, device, getattr(torch, dtype), init=False)
    load_hf(cfg, store, model_dir)
    model = build_model(cfg, store)
    # one partly filled page per sequence, the reserved page, and the tokens themselves
    pages = (max_tokens + page_size - 1) // page_size + max_running + 1
    return Engine(model, max_running=max_running, num_pages=pages, page_size=page_size, max_seq_len=max(max_tokens, 1) + page_size,
                  max_prefill_tokens=max(max_tokens, 1))


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="feed given token ids through a model step by step and write logits")
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for the logits files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live sequences hold at any time")
    ap.add_argument("--device", default="cuda", help="cpu: the PyTorch path of the framework's CPU configuration")
    ns = ap.parse_args(argv)
    import torch

    from ..models import get_config

    if ns.dtype == "float32" and get_config(ns.model).plan is None and ns.device != "cpu":
        print("this model runs in bfloat16 on the GPU", file=sys.stderr)
        return 3
    engine = build_engine(ns.model, ns.dtype, ns.max_tokens, ns.device)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = engine.feed([(e["id"], e["tokens"], e["want"]) for e in step["entries"]])
        wanted = [lg for lg in logits if lg is not None]
        if wanted:
            data = torch.cat(wanted).float().cpu().contiguous().numpy().astype("<f4").tobytes()
            with open(os.path.join(ns.out, f"{step['step']}.f32"), "wb") as f:
                f.write(data)
        if hasattr(engine.model, "check_status"):
            engine.model.check_status()
        for rid in step.get("end", []):
            engine.end_feed(rid)
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
