"""What the tests of checkpoint models share: engines over a test configuration, requests cut into portions, hand-made step plans."""
import json

import numpy as np
import pytest
import torch

from onnx_genai_b200 import replay
from onnx_genai_b200.engine.llm_engine import EngineConfig, LLMEngine
from onnx_genai_b200.models import registry
from onnx_genai_b200.models.decoder import StepInputs
from onnx_genai_b200.package.safetensors import save_file

GPU = pytest.mark.gpu
DEVICES = ["cpu", pytest.param("cuda", marks=GPU)]
ENGINES = [("cpu", "f32"), pytest.param(("cuda", "f32"), marks=GPU), pytest.param(("cuda", "bf16"), marks=GPU)]


def make_engine(cfg, tensors, where, max_tokens=256, max_seqs=4, **kw):
    device, dtype = where
    c = registry.ARCHITECTURES[cfg["architecture"]].read_config(cfg)
    w = registry.ARCHITECTURES[cfg["architecture"]].load_weights(c, tensors, torch.bfloat16 if dtype == "bf16" else torch.float32, device)
    kw = {**dict(num_pages=max_tokens // 16, max_tokens_per_step=max_tokens, prefill_chunk=max_tokens, max_logit_rows=max_tokens,
                 max_seq_len=max_tokens + 16, compute_dtype=dtype), **kw}
    return LLMEngine(EngineConfig(model=c, max_seqs=max_seqs, **kw), weights=w, device=device)


def tokens_of(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def assert_logits(got, want, where, outliers=0.0):
    """Root mean square of every row's difference against the spread of the logits.  The 32-bit engine is the sharp test; in
    bf16 the bound is what rounding leaves in these sharply weighted models, far below what one wrong key or state costs.
    ``outliers``: share of rows that bf16 may leave up to three times further away (designs that norm a head's output, which
    magnifies rounding where that output is next to nothing)."""
    err = (got.double() - want).pow(2).mean(-1).sqrt() / want.std()
    worst, mean = (0.12, 0.04) if where[1] == "bf16" else (1e-4, 2e-5)
    over = (err >= worst).sum() if where[1] == "bf16" and outliers else 0
    top = 3 * worst if over else worst
    assert err.max() < top and over <= max(1.0, outliers * len(err)) and err.mean() < mean, (float(err.max()), float(err.mean()), int(err.argmax()))


def replay_cuts(eng, tokens, cuts, name="a"):
    """Feed one request in portions of the given sizes (the last repeats); logits of every position."""
    rep, at, rows, i = replay.Replayer(eng), 0, [], 0
    while at < len(tokens):
        n = min(cuts[min(i, len(cuts) - 1)], len(tokens) - at)
        rows += rep.step([{"id": name, "tokens": tokens[at:at + n], "want": list(range(n))}], [name] if at + n == len(tokens) else [])
        at, i = at + n, i + 1
    return torch.stack(rows)


def step_of(chunks, device, page_seed=0):
    """A step plan for sequences (tokens before, rows): one-row sequences become decode rows.  Pages are dealt at random."""
    order = [c for c in chunks if c[1] == 1] + [c for c in chunks if c[1] > 1]
    nd = sum(c[1] == 1 for c in chunks)
    mp = max((a + n + 15) // 16 for a, n in order)
    perm = torch.randperm(len(order) * mp, generator=torch.Generator().manual_seed(page_seed)).int().view(len(order), mp)
    slots = torch.randperm(len(order), generator=torch.Generator().manual_seed(page_seed + 1)).int()
    cu, ts, tq, pos, kv = [0], [], [], [], []
    for e, (a, n) in enumerate(order):
        if e >= nd:
            cu.append(cu[-1] + n)
            for q0 in range(0, n, 64):
                ts.append(e - nd)
                tq.append(q0)
        for p in range(a, a + n):
            pos.append(p)
            kv.append(int(perm[e, p // 16]) * 16 + p % 16)
    t = lambda x: torch.tensor(x, dtype=torch.int32, device=device)
    si = StepInputs(len(pos), nd, len(order) - nd, len(ts), 0, token_ids=t([0] * len(pos)), positions=t(pos), slots=t(kv),
                    ctx_len=t([a + n for a, n in order]), page_table=perm.to(device), cu_q=t(cu), tile_seq=t(ts or [0]), tile_q0=t(tq or [0]),
                    logit_rows=t([0]), state_slot=slots.to(device), prefill_ctx=np.array([a + n for a, n in order[nd:]], dtype=np.int32),
                    prefill_len=np.array([n for _, n in order[nd:]], dtype=np.int32))
    return si, order, len(order) * mp


CHUNKS = [(7, 1), (0, 1), (30, 2), (0, 2), (0, 16), (5, 17), (64, 64), (1, 130), (0, 75)]


def write_checkpoint(path, cfg, tensors):
    path.mkdir(exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file(tensors, str(path / "model.safetensors"))
    return str(path)
