"""Replay a trace: feed given token ids through a model step by step and write the logits that were asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N        (also: python -m onnx_genai_b200 replay)

Standard input carries one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every entry's tokens run in that step, all entries as one batch of the engine (the scheduler, caches and kernels that
generation uses; see LLMEngine.open_forced).  ``want`` names places among the tokens; their logits go to OUT/<step>.f32 in
the order of the entries and of ``want`` as little-endian fp32 rows.  Requests in ``end`` give back what they hold.  After
every step a line ``done <step>`` is printed.  The KV pool is made for N tokens and four live requests.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

LIVE = 4              # requests that may be live at a time
STEP_ROWS = 16384     # largest batch of one engine step; a longer step runs as several


def build_engine(model_dir: str, dtype: str, max_tokens: int, device: str):
    from .engine.llm_engine import EngineConfig, LLMEngine
    from .models import registry
    from .ops import PAGE, _native

    doc = registry.native_config(model_dir)
    if doc is None:
        raise SystemExit(f"replay: {model_dir} is not a checkpoint directory of a registered architecture "
                         f"({', '.join(sorted(registry.ARCHITECTURES))})")
    import torch

    kernels = registry.ARCHITECTURES[doc["architecture"]].kernels
    if kernels:
        _native.prefer(kernels)
    f32 = dtype == "float32"
    # fp32 weights on the CPU path (the development statement of the kernels) as everywhere else
    wdtype = torch.float32 if f32 or not device.startswith("cuda") else torch.bfloat16
    cfg, weights = registry.load_checkpoint(model_dir, doc, wdtype, device)
    pages = (max_tokens + 63) // 64 * 64 // PAGE
    rows = min(pages * PAGE, STEP_ROWS)
    ecfg = EngineConfig(model=cfg, num_pages=pages, max_seqs=LIVE, max_tokens_per_step=rows, prefill_chunk=rows, max_logit_rows=rows,
                        max_seq_len=pages * PAGE + PAGE, compute_dtype="f32" if f32 else "bf16")
    return LLMEngine(ecfg, weights=weights, device=device)


class Replayer:
    def __init__(self, engine):
        self.engine, self.open = engine, {}

    def step(self, entries, end):
        """Run the entries' tokens; returns the wanted logits rows (fp32 CPU tensors) in request order."""
        eng, wanted, live = self.engine, [], []
        for e in entries:
            name, tokens, want = e["id"], [int(t) for t in e["tokens"]], [int(k) for k in e.get("want", ())]
            if not tokens:
                continue
            vocab = eng.cfg.model.vocab
            if min(tokens) < 0 or max(tokens) >= vocab:
                raise ValueError(f"request {name}: token ids lie in [0, {vocab})")
            if any(not 0 <= k < len(tokens) for k in want):
                raise ValueError(f"request {name}: 'want' names places outside its {len(tokens)} tokens")
            sid = self.open.get(name)
            start = 0
            if sid is None:
                sid = self.open[name] = eng.open_forced(tokens, want)
            else:
                start = eng.core.seq_len(sid)
                eng.extend_forced(sid, tokens, want)
            live.append(sid)
            wanted += [(sid, start + k) for k in want]
        got = {}
        while any(eng.forced_pending(sid) > 0 for sid in live):
            out = eng.step()
            if out.num_tokens == 0:
                raise RuntimeError("the engine cannot schedule the step: the pool is too small for the live requests")
            for sid, rows in out.forced_logits.items():
                got.update({(sid, pos): row.cpu() for pos, row in rows})
        for name in end:
            eng.close_forced(self.open.pop(name))
        return [got[key] for key in wanted]


def serve(engine, out_dir: str, lines, emit) -> None:
    import torch

    rep = Replayer(engine)
    for line in lines:
        if not line.strip():
            continue
        msg = json.loads(line)
        rows = rep.step(msg["entries"], msg.get("end", ()))
        if rows:
            part = os.path.join(out_dir, f".{msg['step']}.part")
            with open(part, "wb") as f:
                f.write(torch.stack(rows).numpy().astype("<f4").tobytes())
            os.replace(part, os.path.join(out_dir, f"{msg['step']}.f32"))
        emit(f"done {msg['step']}")


def add_arguments(p) -> None:
    p.add_argument("--model", required=True, help="checkpoint directory: config.json and model.safetensors")
    p.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    p.add_argument("--out", required=True, help="directory the logits are written to")
    p.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at a time (each rounded up to 64)")
    p.add_argument("--device", default="cuda", help="cuda[:N]; cpu runs the plain statements of the ops (development only)")


def run(args) -> int:
    engine = build_engine(args.model, args.dtype, args.max_tokens, args.device)
    os.makedirs(args.out, exist_ok=True)

    def emit(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    serve(engine, args.out, sys.stdin, emit)
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    add_arguments(ap)
    return run(ap.parse_args(argv))
