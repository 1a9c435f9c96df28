"""Prefill and decode throughput of hybrid decoders (models/hybrid.py) beside a dense GQA decoder of equal width, depth,
feed-forward and head size, and the row of every kernel against its roofline.  Random weights, synthetic tokens.

    python bench.py --hybrid [--hybrid-sizes small,large] [--hybrid-json out.json]

A step is built by the engine's scheduler and then replayed on the device: prefill steps as the engine launches them (Python
for the hybrid model, the C++ step executor for the dense one), decode steps as CUDA-graph replays for both.  CUDA events
around a few replays, after three warm-up replays; a step's weights and activations exceed the L2 cache.  Kernel rows flush
L2 before every timed launch.
"""
from __future__ import annotations

import json
import sys

import numpy as np
import torch

from .. import ops
from ..engine.core import HDR
from ..engine.llm_engine import EngineConfig, LLMEngine
from ..models.config import DecoderConfig
from ..models.hybrid import HybridConfig, LatentSpec, LayerSpec, MlpSpec, RecurrentSpec
from ..ops import hybrid as hops
from .kernel_bench import Timer, peaks

SIZES = {   # name: hidden, layers, heads (of 128), KV heads of the dense model, feed-forward, latent size, window, streams
    "small": (2048, 16, 16, 4, 8192, 128, 1024, 2),
    "medium": (3072, 12, 24, 8, 8192, 256, 2048, 4),
    "large": (4096, 8, 32, 8, 14336, 512, 4096, 2),
}
VOCAB = 32768


def configs(size: str):
    hid, layers, heads, kvh, ff, rank, window, streams = SIZES[size]
    d = 128
    specs = []
    for i in range(layers):
        if i % 2 == 0:
            mixer = RecurrentSpec(heads, d, d)
        else:
            mixer = LatentSpec(heads, d, d, rank, d ** -0.5, window, kv_from=i - 2 if i % 4 == 3 else None)
        specs.append(LayerSpec(mixer, MlpSpec(ff)))
    hybrid = HybridConfig(vocab=VOCAB, hidden=hid, layers=specs, streams=streams, name=f"rilelorn-{size}")
    dense = DecoderConfig(name=f"dense-{size}", num_layers=layers, hidden=hid, num_heads=heads, num_kv_heads=kvh, head_dim=d, intermediate=ff,
                          vocab=VOCAB, tie_embeddings=False, max_position=16384)
    return hybrid, dense


def build(eng, prompts):
    """One scheduled step for the given requests, its plan on the device."""
    t = eng.core.build_step(eng.plan_host.data_ptr())
    si, hdr = eng.si, eng.plan_np[:32]
    si.num_tokens, si.num_decode = t, int(hdr[HDR["num_decode"]])
    si.num_prefill_seqs, si.num_tiles = int(hdr[HDR["num_prefill_seqs"]]), int(hdr[HDR["num_tiles"]])
    si.num_logit_rows, si.max_ctx = int(hdr[HDR["num_logit_rows"]]), int(hdr[HDR["max_ctx"]])
    eng._host_entries(si)
    eng.plan_dev.copy_(eng.plan_host[: eng.dev_words])
    if si.num_decode:
        eng.model.set_decode_splits(eng._pick_splits(si.num_decode, si.max_ctx))
    return t


def replay_ms(fn, iters=8):
    for _ in range(3):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(iters):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / iters


def run_model(cfg, prefills, decode):
    """{label: (tokens, ms)} for prefill shapes [(requests, tokens each)] and decode (requests, context)."""
    nseq, ctx = decode
    rows = max(max(s * n for s, n in prefills), nseq)
    eng = LLMEngine(EngineConfig(model=cfg, max_seqs=max(nseq, 8), max_tokens_per_step=rows, prefill_chunk=rows, max_seq_len=max(ctx + 64, 8256),
                                 enable_prefix_cache=False, release_window_pages=False), device="cuda")
    rng = np.random.default_rng(0)
    out = {}
    for s, n in prefills:
        ids = [eng.add_request(rng.integers(0, cfg.vocab, n), 4, ignore_eos=True) for _ in range(s)]
        t = build(eng, ids)
        assert t == s * n, (t, s, n)
        out[f"prefill {s} x {n}"] = (t, replay_ms(lambda: eng.model.forward(eng.si, eng.kv), iters=5))
        for i in ids:
            eng.core.release(i)
    ids = [eng.add_request(rng.integers(0, cfg.vocab, ctx), 64, ignore_eos=True) for _ in range(nseq)]
    while any(eng.core.seq_computed(i) < ctx for i in ids):
        eng.step()
    t = build(eng, ids)
    assert eng.si.num_decode == t
    fwd = lambda: eng.model.forward(eng.si, eng.kv)
    fwd()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g, capture_error_mode="thread_local"):
        fwd()
    out[f"decode {t} rows, context {ctx}"] = (t, replay_ms(g.replay, iters=20))
    eng.check_device_status()
    return out


def _plan(chunks, max_pages, num_pages):
    """StepInputs of sequences (tokens before, rows), one-row sequences first, pages in order."""
    from ..models.decoder import StepInputs

    nd = sum(n == 1 for _, n in chunks)
    cu, ts, tq, slots, table, nxt = [0], [], [], [], [], 0
    for e, (a, n) in enumerate(chunks):
        np_ = (a + n + 15) // 16
        pages = [(nxt + k) % num_pages for k in range(np_)]
        nxt += np_
        table.append(pages + [0] * (max_pages - np_))
        slots += [pages[p // 16] * 16 + p % 16 for p in range(a, a + n)]
        if e >= nd:
            cu.append(cu[-1] + n)
            for q0 in range((n - 1) // 64 * 64, -1, -64):
                ts.append(e - nd)
                tq.append(q0)
    t = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
    pos = [p for a, n in chunks for p in range(a, a + n)]
    return StepInputs(len(pos), nd, len(chunks) - nd, len(ts), 0, token_ids=t([0] * len(pos)), positions=t(pos), slots=t(slots),
                      ctx_len=t([a + n for a, n in chunks]), page_table=t(table), cu_q=t(cu), tile_seq=t(ts or [0]), tile_q0=t(tq or [0]),
                      logit_rows=t([0]), state_slot=t(list(range(len(chunks)))), prefill_ctx=np.array([a + n for a, n in chunks[nd:]], dtype=np.int32),
                      prefill_len=np.array([n for _, n in chunks[nd:]], dtype=np.int32))


def seen_pairs(chunks, window):
    tot = 0
    for a, n in chunks:
        pos = np.arange(a, a + n) + 1
        tot += int(np.minimum(pos, window).sum() if window > 0 else pos.sum())
    return tot


def kernel_rows(size: str, timer, pk):
    """One row per kernel: the hybrid model's beside the like kernel of the dense model, at this size's shapes."""
    hid, _, heads, kvh, ff, rank, window, streams = SIZES[size]
    d, bf = 128, torch.bfloat16
    rnd = lambda *s, dtype=bf: (torch.randn(*s, device="cuda") * 0.1).to(dtype)
    rows = []

    def row(name, phase, fn, flops=0, nbytes=0):
        ms, _ = timer.time(fn)
        bound = max(flops / (pk["bf16_tflops"] * 1e12), nbytes / (pk["hbm_gbs"] * 1e9)) * 1e3
        rows.append({"kernel": name, "step": phase, "ms": round(ms, 4), "roofline_ms": round(bound, 4), "of_roofline": round(bound / ms, 3),
                     "TF/s": round(flops / ms / 1e9, 1) if flops else None, "GB/s": round(nbytes / ms / 1e6, 1) if nbytes else None})

    for phase, chunks in (("prefill 4096", [(0, 4096)]), ("prefill 4x1024", [(0, 1024)] * 4), ("decode 64", [(2047, 1)] * 64), ("decode 64, context 8192", [(8191, 1)] * 64)):
        t, nseq = sum(n for _, n in chunks), len(chunks)
        ctx = max(a + n for a, n in chunks)
        mp, npages = (ctx + 15) // 16, sum((a + n + 15) // 16 for a, n in chunks)
        si = _plan(chunks, mp, npages)
        x0, x1 = rnd(t, streams, hid, dtype=torch.float32), torch.empty(t, streams, hid, device="cuda")
        y, h = rnd(t, hid), torch.empty(t, hid, dtype=bf, device="cuda")
        f32 = lambda *s: torch.rand(*s, device="cuda")
        conn, norm = hops.HyperConnection(f32(streams), f32(streams), f32(streams, streams)), hops.DynamicTanh(f32(1), f32(hid), f32(hid))
        xb = t * streams * hid * 4
        row("hyper_step", phase, lambda: hops.hyper_step(x0, x1, y, conn, conn.read, norm, h, si), nbytes=2 * xb + 2 * t * hid * 2)
        prev, amount = f32(nseq, hid), f32(hid)
        row("hyper_step + shift", phase, lambda: hops.hyper_step(x0, x1, y, conn, conn.read, norm, h, si, shift=amount, prev=prev),
            nbytes=2 * xb + 2 * t * hid * 2)
        w1 = torch.ones(hid, device="cuda", dtype=bf)
        row("dense: rmsnorm", phase, lambda: ops.rmsnorm(y, w1, 1e-6, out=h), nbytes=2 * t * hid * 2)
        # recurrence
        n_qfv = heads * 3 * d
        wq, qfv = rnd(n_qfv, hid), torch.empty(t, n_qfv, device="cuda")
        row("gemm q|f|v (fp32 out)", phase, lambda: hops.linear(h, wq, qfv, f32_out=True), 2 * t * n_qfv * hid, (n_qfv + t) * hid * 2 + t * n_qfv * 4)
        qfv.normal_()
        state, raw = torch.zeros(nseq, heads, d, d, device="cuda"), torch.empty(t, heads * d, device="cuda")
        bias, low = f32(heads * d) * 2, f32(heads * d) * 0.5
        row("hgrn2", phase, lambda: hops.hgrn2(qfv, bias, low, state, raw, heads, d, d, si, split=True), nbytes=t * heads * d * 16 + 2 * nseq * heads * d * d * 4)
        nw, attn = f32(d), torch.empty(t, heads * d, dtype=bf, device="cuda")
        row("head_rmsnorm", phase, lambda: hops.head_rmsnorm(raw, nw, 1e-6, attn, heads, d), nbytes=t * heads * d * 6)
        if phase.startswith("prefill"):
            from ..ops import sequence

            b, tt = nseq, t // nseq
            la = lambda: sequence.linear_attention(rnd_q, rnd_q, rnd_q, past, dec, None, heads, heads, "gated", 1.0)
            rnd_q, past, dec = rnd(b, tt, heads * d), torch.zeros(b, heads, d, d, dtype=bf, device="cuda"), -rnd(b, tt, heads * d).abs()
            row("graph operator: linear_attention (gated)", phase, la, nbytes=t * heads * d * 10 + 2 * b * heads * d * d * 2)
        # latent attention
        c, wn, pool = rnd(t, rank), f32(rank), rnd(npages, 16, rank)
        row("latent_append", phase, lambda: hops.latent_append(c, 0, wn, 1e-6, si.slots, pool, rank), nbytes=2 * t * rank * 2)
        q, uk, qa, oc = rnd(t, heads * d), rnd(heads * rank, d), rnd(t, heads * rank), torch.empty(t, heads * rank, dtype=bf, device="cuda")
        uv, o = rnd(heads * d, rank), torch.empty(t, heads * d, dtype=bf, device="cuda")
        wb = heads * rank * d * 2
        row("gemm per head (W_uk^T q)", phase, lambda: hops.linear_batched(q, uk, qa, heads, d, rank), 2 * t * heads * d * rank, t * heads * (d + rank) * 2 + wb)
        row("gemm per head (W_uv o)", phase, lambda: hops.linear_batched(oc, uv, o, heads, rank, d), 2 * t * heads * d * rank, t * heads * (d + rank) * 2 + wb)
        qa = rnd(t * heads, rank)
        oc = torch.empty_like(qa)
        pairs, keys = seen_pairs(chunks, window), sum(min(a + n, window + n) for a, n in chunks)
        if si.num_prefill_seqs:
            row("latent_attention (latents as keys)", phase, lambda: hops.latent_attention(qa, oc, pool, si, heads, rank, 0.1, window),
                4 * pairs * heads * rank, keys * rank * 2 + 2 * t * heads * rank * 2)
            if rank > d:      # what prompts of this shape run on
                pages = hops.visible_pages(si, window)
                dense, kvp = torch.empty(pages * 16, rank, dtype=bf, device="cuda"), torch.empty(pages, heads, 2 * d // 64, 16, 64, dtype=bf, device="cuda")
                table, kvw, qd = torch.zeros(nseq, mp, dtype=torch.int32, device="cuda"), rnd(heads * 2 * d, rank), rnd(t, heads * d)
                od = torch.empty(t, heads * d, dtype=bf, device="cuda")
                row("latent prompt, expanded K/V (3 kernels)", phase, lambda: hops.latent_prefill_expanded(qd, od, pool, kvw, si, heads, d // 64, d // 64, d, d, 0.1,
                                                                                                          window, pages, dense, kvp, table),
                    4 * pairs * heads * d + 2 * pages * 16 * rank * heads * 2 * d, 2 * pages * 16 * heads * 2 * d * 2)
        else:
            cnt = torch.zeros(4096, dtype=torch.int32, device="cuda")
            splits = max(1, 148 * (2 if rank <= 128 else 1) // nseq // 2 * 2)
            po, pm = torch.empty(t * heads * splits * rank, device="cuda"), torch.empty(t * heads * splits * 2, device="cuda")
            row(f"latent_attention (decode, {splits} splits)", phase, lambda: hops.latent_attention(qa, oc, pool, si, heads, rank, 0.1, window, splits, po,
                                                                                                   pm, cnt),
                4 * pairs * heads * rank, keys * rank * 2 + 2 * t * heads * rank * 2)
        # the dense model's attention and projections
        nq = (heads + 2 * kvh) * d
        qkv, out, kv = rnd(t, nq), torch.empty(t, heads * d, dtype=bf, device="cuda"), rnd(npages, kvh, 2, 16, d)
        allp = seen_pairs(chunks, 0)
        if si.num_prefill_seqs:
            row("dense: paged_prefill", phase, lambda: ops.paged_prefill(qkv, out, kv, si.page_table, si.ctx_len, si.cu_q, si.tile_seq, si.tile_q0,
                                                                          si.num_tiles, heads, kvh, d), 4 * allp * heads * d, t * (nq + heads * d) * 2)
        else:
            row("dense: paged_decode", phase, lambda: ops.paged_decode(qkv, out, kv, si.page_table, si.ctx_len, heads, kvh, d), 4 * allp * heads * d,
                allp * kvh * 2 * d * 2)
        wqkv = rnd(nq, hid)
        row("dense: gemm qkv", phase, lambda: ops.gemm(h, wqkv, out=qkv), 2 * t * nq * hid, (nq + t) * hid * 2 + t * nq * 2)
        # feed-forward
        gu, act = rnd(2 * ff, hid), torch.empty(t, ff, dtype=bf, device="cuda")
        fl, by = 4 * t * ff * hid, (2 * ff + t) * hid * 2 + t * ff * 2
        row("gemm gate_up (gelu gate)", phase, lambda: hops.gated_linear(h, gu, 128, "gelu_tanh", act), fl, by)
        row("dense: gemm gate_up (silu gate)", phase, lambda: ops.gemm(h, gu, epilogue="swiglu", swiglu_half=128, out=act), fl, by)
        dn, res = rnd(hid, ff), rnd(t, hid)
        fl, by = 2 * t * ff * hid, (ff + t) * hid * 2 + t * ff * 2
        row("gemm down", phase, lambda: hops.linear(act, dn, y), fl, by)
        row("dense: gemm down (+ residual)", phase, lambda: ops.gemm(act, dn, residual=res, epilogue="residual", out=res), fl, by)
    ops.check_status()
    return rows


def main(sizes, json_path="") -> dict:
    pk, timer = peaks(), Timer()
    doc = {"peaks": pk, "sizes": {}}
    for size in sizes:
        hybrid, dense = configs(size)
        prefills, decode = [(1, 4096), (4, 1024)], (64, 2048)
        res = {"hybrid": run_model(hybrid, prefills, decode)}
        torch.cuda.empty_cache()
        res["dense"] = run_model(dense, prefills, decode)
        torch.cuda.empty_cache()
        doc["sizes"][size] = {"config": SIZES[size], "weights_gb": {"hybrid": hybrid.weight_bytes() / 1e9, "dense": dense.weight_bytes() / 1e9},
                              "throughput": {m: {k: {"ms": round(ms, 3), "tok_s": round(t / ms * 1e3)} for k, (t, ms) in r.items()} for m, r in res.items()},
                              "kernels": kernel_rows(size, timer, pk)}
        print(f"== {size} {SIZES[size]}", file=sys.stderr)
        for m, r in doc["sizes"][size]["throughput"].items():
            for k, v in r.items():
                print(f"  {m:7s} {k:28s} {v['ms']:9.3f} ms {v['tok_s']:>9d} tok/s", file=sys.stderr)
        for r in doc["sizes"][size]["kernels"]:
            print(f"  {r['step']:15s} {r['kernel']:42s} {r['ms']:8.4f} ms  roofline {r['roofline_ms']:8.4f}  {r['of_roofline']:.3f}  "
                  f"{r['TF/s'] or '':>7} TF/s {r['GB/s'] or '':>8} GB/s", file=sys.stderr)
    if json_path:
        with open(json_path, "w", encoding="utf-8") as f:
            json.dump(doc, f, indent=1)
    return doc
