"""Command line of the trace replayer: ``bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N``.

Reads one JSON object a line from standard input, ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``,
runs each as one engine step (:class:`.replay.TraceReplayer`), writes the wanted logits to ``DIR/<step>.f32``
(little-endian fp32 ``[wanted, vocab]``) and prints ``done <step>`` after every step. The kernels a model family needs
are compiled first if no current library is there.
"""

from __future__ import annotations

import argparse
import json
import os
import sys

MAX_REQUESTS = 4


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replays a token trace through the serving engine.")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="where <step>.f32 files go")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="most tokens live requests hold together (sizes the page pool)")
    ap.add_argument("--max-requests", type=int, default=MAX_REQUESTS, help="most live requests (state slots)")
    args = ap.parse_args(argv)

    from ...csrc.build import ensure
    from ...infra.factory import TaskType, _ensure_models_imported, registry

    _ensure_models_imported()
    with open(os.path.join(args.model, "config.json"), encoding="utf-8") as f:
        model_type = registry.model_type_of(json.load(f))
    module = registry.get_module_registration(TaskType.CAUSAL_LM, model_type).module
    import torch

    if torch.cuda.is_available():
        from ...ops import _lib

        _lib.use_library(ensure(model_type))
    from ...caching.paged import PAGE_SIZE
    from .engine import eSurge
    from .replay import TraceReplayer, engine_limits

    model = module.from_pretrained(args.model, dtype=getattr(torch, args.dtype))
    engine = eSurge(model, enable_prefix_caching=False, async_scheduling=False,
                    **engine_limits(args.max_tokens, args.max_requests, PAGE_SIZE))
    replay = TraceReplayer(engine)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step.get("entries", ()), step.get("end", ()))
        if logits is not None:
            path = os.path.join(args.out, f"{step['step']}.f32")
            logits.contiguous().numpy().astype("<f4").tofile(path)
        print(f"done {step['step']}", flush=True)
    engine.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
