"""Feed given token ids through a model step by step and write logits (``bin/trace_run``).

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A line of the input is one step: ``{"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}``.
All entries of a step are one batch.  A step in which something is wanted leaves ``OUT/<step>.f32``: the logits at the wanted
places in the order of the entries, little-endian fp32 ``[wanted, vocab]``.  After every step ``done <step>`` is printed.
Requests listed in ``end`` give back their pages and slot after the step.

The engine is the serving one: checkpoint admission and model class by ``config.json``, scheduler, page pool for ``N`` tokens,
four request slots, the native runner and its decode graphs.  In a fresh checkout the first call compiles the kernels that the model
needs.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

MAX_LIVE_REQUESTS = 4


def build_engine(model: str, dtype: str, max_tokens: int, device: int = 0, max_requests: int = MAX_LIVE_REQUESTS):
    """An engine for a checkpoint directory whose cache holds ``max_tokens`` tokens (plus the pool's reserved page)."""
    import torch

    from ..executor.gpu_executor import GpuExecutor
    from ..models import registry
    from ..models.checkpoint import admit_checkpoint
    from ..runtime.engine import LLMEngine
    from ..runtime.scheduler import SchedulerConfig
    ck = admit_checkpoint(model)
    if ck.cfg.family == "layered":
        from ..models.layered import with_dtype
        ck.cfg = with_dtype(ck.cfg, dtype)
    elif dtype != "bfloat16":
        raise SystemExit(3)                      # the quantized decoders compute in 16 bits on the GPU
    dev = torch.device("cuda", device)
    torch.cuda.set_device(dev)
    defn = registry.get(ck.cfg.family)
    pages = -(-max_tokens // 16) + 1
    runner = defn.build_runner(ck.cfg, defn.load_weights(ck, dev), num_pages=pages, max_tokens=max(16, max_tokens),
                               max_requests=max_requests)
    ex = GpuExecutor(runner, max_rows=max_requests, max_prefill_tokens=max(16, max_tokens), max_model_len=max(16, max_tokens))
    ex.capture_decode_graphs()
    return LLMEngine(ex, num_pages=pages, scheduler_config=SchedulerConfig(
        max_running_requests=max_requests, max_batched_tokens=max(16, max_tokens), max_model_len=max(16, max_tokens),
        enable_prefix_cache=False))


def run(session, lines, out: Path, stdout=sys.stdout) -> None:
    import numpy as np
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        got = session.step([(str(e["id"]), e["tokens"], e.get("want") or []) for e in step["entries"]]) if step["entries"] else []
        if sum(len(g) for g in got):
            np.concatenate(got).astype("<f4").tofile(out / f"{int(step['step'])}.f32")
        session.end(str(i) for i in step.get("end") or ())
        print(f"done {int(step['step'])}", file=stdout, flush=True)


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="feed token ids through a model step by step, write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at most")
    ap.add_argument("--device", type=int, default=0)
    args = ap.parse_args(argv)
    from ..models.checkpoint import layered_config_of
    from ..models.layered import kernel_sources
    from ..ops import native
    from ..runtime.imposed import ImposedSession
    layered = layered_config_of(Path(args.model))
    if layered is not None:
        native.select(kernel_sources(layered))       # a checkout without the library compiles what this model needs
    engine = build_engine(args.model, args.dtype, args.max_tokens, args.device)
    out = Path(args.out)
    out.mkdir(parents=True, exist_ok=True)
    run(ImposedSession(engine), iter(sys.stdin.readline, ""), out)
    engine.executor.runner.ws.check_status()
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
