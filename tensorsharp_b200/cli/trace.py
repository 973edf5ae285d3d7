"""``bin/trace_run``: feed given token ids through a model and write the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Every line of standard input is one step, ``{"step": 7, "entries": [{"id": "x", "tokens": [31, 8], "want": [1]}], "end": ["y"]}``:
the entries are one batch of the engine (portions of prompts beside single tokens; ``want``: places among the entry's tokens
whose logits are wanted), the requests of ``end`` give their pages and slot back afterwards.  The wanted logits go to
``DIR/<step>.f32`` (little-endian float32, [wanted, vocab]); ``done <step>`` is printed after every step.  Nothing is
sampled; admission, pages, batches and kernels are those of generation (runtime/batching.py: StepEngine).

The cache pool holds ``--max-tokens`` tokens, and four requests may be live.  On a machine where the kernel library has not
been built, the first call compiles the sources that the model's family needs.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import List, Optional

MAX_LIVE = 4
EXIT_NO_FLOAT32 = 3


def write_logits(path: str, logits) -> None:
    data = logits.detach().to("cpu").float().contiguous().numpy().astype("<f4", copy=False).tobytes()
    with open(path + ".part", "wb") as f:
        f.write(data)
    os.replace(path + ".part", path)


def run_steps(model, lines, out_dir: str, emit=print) -> None:
    from ..runtime.batching import StepEngine
    eng = StepEngine(model, MAX_LIVE)
    vocab = model.cfg.vocab
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [(e["id"], e["tokens"], e.get("want") or []) for e in step["entries"]]
        for key, tokens, _ in entries:
            if any(not 0 <= int(t) < vocab for t in tokens):
                raise ValueError(f"step {step['step']}: request {key!r} has a token id outside [0, {vocab})")
        logits = eng.step(entries) if entries else None
        if logits is not None:
            write_logits(os.path.join(out_dir, f"{step['step']}.f32"), logits[:, :vocab])
        for key in step.get("end") or []:
            eng.end(key)
        model.poll_status(force=True)                     # a kernel's bounded wait that gave up ends the run with an error
        emit(f"done {step['step']}")


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="model folder (config.json, model.safetensors) or GGUF file")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default="cuda", help="cuda, or cpu for the reference ops (float32)")
    a = ap.parse_args(argv)
    import torch

    from ..models.base import ModelBase
    from ..ops import native
    cls = ModelBase.class_of(a.model)
    on_gpu = a.device.startswith("cuda")
    if on_gpu and a.dtype == "float32" and not cls.supports_float32:
        print(f"error: {cls.__name__} has no float32 path", file=sys.stderr)
        return EXIT_NO_FLOAT32
    if on_gpu:
        if not torch.cuda.is_available():
            raise RuntimeError("no CUDA device")
        native.ensure(cls.native_sources)
    page = 64
    pages = (max(1, a.max_tokens) + page - 1) // page
    os.makedirs(a.out, exist_ok=True)
    model = ModelBase.create(a.model, a.device, max_context=pages * page, max_seqs=MAX_LIVE, page_size=page, kv_pages=pages,
                             compute_dtype=getattr(torch, a.dtype) if on_gpu else None)
    try:
        with torch.inference_mode():
            run_steps(model, sys.stdin, a.out, emit=lambda text: print(text, flush=True))
    finally:
        model.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
