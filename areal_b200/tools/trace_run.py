"""Trace runner: feeds given token ids through a served model, step by step, and writes the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A step is one line ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``: every entry brings the next
tokens of its request, all entries run as one batch, ``want`` are the places among the tokens whose logits go to
``DIR/<n>.f32`` (little-endian fp32, in order). ``done <n>`` is printed after every step; requests under ``end`` give
their pages and state slot back. Nothing is sampled: the steps run on the rollout engine's own model, cache and step
function (:class:`~areal_b200.engine.ragged_step.RaggedRunner`), with a pool of ``N`` tokens and four state slots.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE_SIZE = 64
SLOTS = 4


def make_engine(model: str, dtype: str, max_tokens: int, device: str = "cuda"):
    from ..api.cli_args import InferenceEngineConfig, NativeInferConfig
    from ..engine.infer_engine import NativeInferenceEngine
    from ..models.config import ModelConfig

    cfg = ModelConfig.from_pretrained(model)
    if not cfg.is_mixer_stack:
        raise SystemExit(f"{cfg.arch}: only models that run by ragged steps (mixer stacks) can replay a trace")
    ic = NativeInferConfig(page_size=PAGE_SIZE, num_pages=max(1, -(-max_tokens // PAGE_SIZE)), max_running_requests=SLOTS,
                           context_length=max(max_tokens, PAGE_SIZE), compute_dtype=dtype)
    return NativeInferenceEngine(InferenceEngineConfig(), ic, model_config=cfg).initialize(
        device=device, model_path=model, start_executor=False, start_loop=False)


def replay(engine, lines, out_dir: str, emit) -> None:
    """Runs the steps of ``lines`` (JSON texts) and calls ``emit("done <n>")`` after each."""
    import contextlib

    import torch

    from ..engine.ragged_step import Entry

    live: dict = {}
    cache = engine.cache
    on_stream = (lambda: torch.cuda.stream(engine.stream)) if engine.device.type == "cuda" else contextlib.nullcontext
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = cache.open()
                if live[e["id"]] is None:
                    raise RuntimeError(f"more than {cache.num_slots} requests are live")
            c = live[e["id"]]
            if not cache.grow(c, c.length + len(e["tokens"])):
                raise RuntimeError("live requests hold more tokens than the pool was made for")
            entries.append(Entry(c, e["tokens"], e["want"]))
        if entries:
            with on_stream():
                logits = engine.runner.step(entries)
                if logits is not None:
                    data = logits.float().contiguous().cpu().numpy().astype("<f4").tobytes()
                    with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                        f.write(data)
                if engine.device.type == "cuda":
                    engine._err_poll.enqueue()
                    engine.stream.synchronize()
                    engine._err_poll.check("trace step")
        for rid in step.get("end", []):
            cache.close(live.pop(rid))
        emit(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay tokens through a model, write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    a = ap.parse_args(argv)
    import torch

    if not torch.cuda.is_available():
        print("trace_run needs a CUDA device", file=sys.stderr)
        return 1
    from ..models.config import ModelConfig
    from ..models.mixers import DESIGNS
    from ..ops import build as kbuild
    from ..ops import lib as oplib

    cfg = ModelConfig.from_pretrained(a.model)
    if cfg.is_mixer_stack:
        oplib.use_library(kbuild.build_step_library(cfg.arch, DESIGNS[cfg.arch].kernels))
    torch.cuda.set_device(0)
    os.makedirs(a.out, exist_ok=True)
    engine = make_engine(a.model, a.dtype, a.max_tokens)
    replay(engine, sys.stdin, a.out, lambda s: print(s, flush=True))
    return 0


if __name__ == "__main__":
    sys.exit(main())
