"""Prefill and decode throughput of delta-rule / differential-attention decoders with routed experts (models/dezudra.py) beside a GQA
decoder with as many experts of equal width, depth, heads and expert size, and the row of every kernel beside the like kernel of
the existing models.  Random weights, synthetic tokens; steps and timing as in :mod:`.hybrid_bench`.

    python bench.py --hybrid --hybrid-design dezudra [--hybrid-sizes small,large] [--hybrid-json out.json]
"""
from __future__ import annotations

import json
import sys

import torch

from .. import ops
from ..models.config import DecoderConfig, MoEConfig
from ..models.hybrid import DeltaSpec, DiffSpec, HybridConfig, LayerSpec, MoeSpec
from ..ops import hybrid as hops
from ..ops import moe as mops
from .hybrid_bench import VOCAB, _plan, run_model
from .kernel_bench import Timer, peaks

# hidden, layers, attention heads / KV heads (two maps of dim, values of 128), dim, window, kept first tokens, delta heads / key heads (of 128),
# experts, chosen, groups, groups kept, expert feed-forward
SIZES = {
    "small": (2048, 12, 16, 4, 64, 1024, 64, 16, 8, 32, 4, 4, 2, 1024),
    "medium": (3072, 9, 24, 8, 64, 2048, 100, 24, 12, 64, 6, 8, 4, 1024),
    "large": (4096, 6, 32, 8, 128, 4096, 128, 32, 16, 16, 2, 4, 2, 4096),
}
DV = 128          # value width of attention heads, both widths of delta heads
TAPS = 4


def configs(size: str):
    hid, layers, hq, hkv, d, window, keep, dh, dg, e, top, groups, kept, ff = SIZES[size]
    moe = MoeSpec(e, top, ff, groups, kept)
    specs = [LayerSpec(DeltaSpec(dh, dg, DV, DV, TAPS) if i % 3 == 2 else
                       DiffSpec(hq, hkv, d, DV, TAPS, d ** -0.5, 0.5, window, keep, d // 2, 5e4), moe) for i in range(layers)]
    new = HybridConfig(vocab=VOCAB, hidden=hid, layers=specs, residual="sandwich", name=f"dezudra-{size}")
    like = DecoderConfig(name=f"moe-{size}", num_layers=layers, hidden=hid, num_heads=hq, num_kv_heads=hkv, head_dim=DV, intermediate=0, vocab=VOCAB,
                         tie_embeddings=False, max_position=16384, moe=MoEConfig(num_experts=e, top_k=top, expert_intermediate=ff))
    return new, like


def visible_pairs(chunks, window, keep):
    """(query, key) pairs inside the mask, and keys that some query of a sequence sees."""
    pairs = keys = 0
    for a, n in chunks:
        for p in range(a, a + n):
            lo = max(0, p - window + 1) if window > 0 else 0
            pairs += p + 1 - lo + min(keep, lo)
        lo = max(0, a - window + 1) if window > 0 else 0
        keys += a + n - lo + min(keep, lo)
    return pairs, keys


def kernel_rows(size: str, timer, pk):
    """One row per kernel: this design's, and behind it the like kernel of the existing models ("like: ...") at the same shapes."""
    hid, _, hq, hkv, d, window, keep, dh, dg, e, top, groups, kept, ff = SIZES[size]
    bf = torch.bfloat16
    rnd = lambda *s, dtype=bf: (torch.randn(*s, device="cuda") * 0.1).to(dtype)
    f32 = lambda *s: torch.rand(*s, device="cuda")
    empty = lambda *s, dtype=bf: torch.empty(*s, dtype=dtype, device="cuda")
    rows = []

    def row(name, phase, fn, flops=0, nbytes=0):
        ms, _ = timer.time(fn)
        bound = max(flops / (pk["bf16_tflops"] * 1e12), nbytes / (pk["hbm_gbs"] * 1e9)) * 1e3
        rows.append({"kernel": name, "step": phase, "ms": round(ms, 4), "roofline_ms": round(bound, 4), "of_roofline": round(bound / ms, 3),
                     "TF/s": round(flops / ms / 1e9, 1) if flops else None, "GB/s": round(nbytes / ms / 1e6, 1) if nbytes else None})

    for phase, chunks in (("prefill 4096", [(0, 4096)]), ("prefill 4x1024", [(0, 1024)] * 4), ("decode 64", [(2047, 1)] * 64),
                          ("decode 64, context 8192", [(8191, 1)] * 64)):
        t, nseq = sum(n for _, n in chunks), len(chunks)
        ctx = max(a + n for a, n in chunks)
        mp, npages = (ctx + 15) // 16, sum((a + n + 15) // 16 for a, n in chunks)
        si = _plan(chunks, mp, npages)
        prompt = si.num_prefill_seqs > 0
        # norms and residual
        x, y, h = rnd(t, hid, dtype=torch.float32), rnd(t, hid), empty(t, hid)
        w, w1 = hops.RmsNorm(f32(hid), 1e-6), torch.ones(hid, device="cuda", dtype=bf)
        row("norm_step", phase, lambda: hops.norm_step(x, y, w, w, h), nbytes=t * hid * (8 + 4))
        routed = hops.ExpertRows(rnd(t * top, hid), torch.randperm(t * top, device="cuda").int().view(t, top), f32(t, top))
        row("norm_step over expert rows", phase, lambda: hops.norm_step(x, routed, w, w, h), nbytes=t * hid * (8 + 2 + 2 * top))
        row("like: rmsnorm with residual delta", phase, lambda: ops.rmsnorm(h, w1, 1e-6, delta=y, out=y), nbytes=t * hid * 8)
        lib, st = ops._native.load(), torch.cuda.current_stream().cuda_stream
        tw = f32(t, top)
        row("like: moe_combine", phase, lambda: lib.ogb_moe_combine(routed.rows.data_ptr(), routed.pos.data_ptr(), tw.data_ptr(), h.data_ptr(), t, top, hid, 1, st),
            nbytes=t * hid * (4 + 2 * top))
        # attention
        n = (2 * hq + 2 * hkv) * d + hkv * DV
        wqkv, u, q, attn = rnd(n, hid), empty(t, n), empty(t, 2 * hq * d), empty(t, hq * DV)
        pool = rnd(npages, 16 * hkv * (2 * d + DV))
        row("gemm q|k|v", phase, lambda: hops.linear(h, wqkv, u), 2 * t * n * hid, (n + t) * hid * 2 + t * n * 2)
        u.normal_()
        conv, bias, state = f32(TAPS, n), f32(n), torch.zeros(nseq, TAPS - 1, n, device="cuda")
        freq = torch.rand(d // 4, dtype=torch.float64, device="cuda")
        row("conv_rope_append", phase, lambda: hops.conv_rope_append(u, conv, bias, state, q, pool, freq, si, 2 * hq, 2 * hkv, hkv, d, DV, d, DV),
            nbytes=2 * t * n * 2 + 2 * nseq * (TAPS - 1) * n * 4)
        pairs, keys = visible_pairs(chunks, window, keep)
        fl, by = 2 * pairs * hq * 2 * (d + DV), keys * hkv * (2 * d + DV) * 2 + t * hq * (2 * d + DV) * 2
        qkv, out, kv = rnd(t, (hq + 2 * hkv) * DV), empty(t, hq * DV), rnd(npages, hkv, 2, 16, DV)
        table = ops.reference.rope_table(ctx + 1, DV, 1e4, "cuda")
        row("like: rope_kv_append", phase, lambda: ops.rope_kv_append(qkv, si.positions, si.slots, table, kv, hq, hkv, DV), nbytes=2 * t * (hq + 2 * hkv) * DV * 2)
        lfl, lby = 4 * pairs * hq * DV, keys * hkv * 2 * DV * 2 + 2 * t * hq * DV * 2
        sink = (keep + 15) // 16 * 16
        if prompt:
            row("diff_attention (prompt)", phase, lambda: hops.diff_attention(q, attn, pool, si, hq, hkv, d, DV, d, DV, d ** -0.5, 0.5, 1e-6, 0.5, window, keep), fl, by)
            row("like: paged_prefill (window and sinks)", phase, lambda: ops.paged_prefill(qkv, out, kv, si.page_table, si.ctx_len, si.cu_q, si.tile_seq, si.tile_q0,
                                                                                         si.num_tiles, hq, hkv, DV, None, window, sink=sink), lfl, lby)
            row("like: paged_prefill (window, tcgen05)", phase, lambda: ops.paged_prefill(qkv, out, kv, si.page_table, si.ctx_len, si.cu_q, si.tile_seq, si.tile_q0,
                                                                                        si.num_tiles, hq, hkv, DV, None, window), lfl, lby)
        else:
            ctas = hkv * -(-(hq // hkv) // 8)
            splits = 1
            while 2 * splits * ctas * nseq <= 296 and min(ctx, window) // (2 * splits) >= 128:
                splits *= 2
            cnt = torch.zeros(nseq * ctas, dtype=torch.int32, device="cuda")
            po, pm = empty(nseq * ctas * 16 * splits * DV, dtype=torch.float32), empty(nseq * ctas * 32 * splits, dtype=torch.float32)
            row(f"diff_attention (decode, {splits} splits)", phase, lambda: hops.diff_attention(q, attn, pool, si, hq, hkv, d, DV, d, DV, d ** -0.5, 0.5, 1e-6, 0.5, window,
                                                                                               keep, splits, po, pm, cnt), fl, by)
            row("like: paged_decode (window and sinks)", phase, lambda: ops.paged_decode(qkv, out, kv, si.page_table, si.ctx_len, hq, hkv, DV, None, 1, None, None, window,
                                                                                        sink=sink), lfl, lby)
        wo = rnd(hid, hq * DV)
        row("gemm o", phase, lambda: hops.linear(attn, wo, y), 2 * t * hid * hq * DV, (hid + t) * hq * DV * 2 + t * hid * 2)
        wl = rnd((hq + 2 * hkv) * DV, hid)
        row("like: gemm qkv", phase, lambda: ops.gemm(h, wl, out=qkv), 2 * t * wl.shape[0] * hid, (wl.shape[0] + t) * hid * 2 + t * wl.shape[0] * 2)
        # delta rule
        c = (2 * dg + dh) * DV
        wd, wab, ud, ab = rnd(c + dh * DV, hid), rnd(2 * dh, hid), empty(t, c + dh * DV), empty(t, 2 * dh, dtype=torch.float32)
        row("gemm gate|q|k|v", phase, lambda: hops.linear(h, wd, ud), 2 * t * wd.shape[0] * hid, (wd.shape[0] + t) * hid * 2 + t * wd.shape[0] * 2)
        row("gemm decay|step (fp32 out)", phase, lambda: hops.linear(h, wab, ab, f32_out=True), 2 * t * 2 * dh * hid, (2 * dh + t) * hid * 2 + t * 2 * dh * 4)
        ud.normal_()
        cd, sd = f32(TAPS, c), torch.zeros(nseq, TAPS - 1, c, device="cuda")
        qk, v, gates = empty(t, 2 * dg * DV, dtype=torch.float32), empty(t, dh * DV), empty(t, dh, 2, dtype=torch.float32)
        al, dt = -f32(dh), f32(dh) - 3
        row("conv_unit_gates", phase, lambda: hops.conv_unit_gates(ud[:, dh * DV:], cd, sd, ab, al, dt, qk, v, gates, si, dg, dh, DV, DV),
            nbytes=t * (c * 2 + 2 * dg * DV * 4 + dh * DV * 2 + dh * 16) + 2 * nseq * (TAPS - 1) * c * 4)
        rec, raw = torch.zeros(nseq, dh, DV, DV, device="cuda"), empty(t, dh * DV, dtype=torch.float32)
        work: dict = {}

        def scratch(name, shape):
            if name not in work:
                work[name] = empty(*shape, dtype=torch.float32)
            return work[name]

        row("delta_rule", phase, lambda: hops.delta_rule(qk, v, gates, rec, raw, dh, dg, DV, DV, si, blocks=True, scratch=scratch),
            nbytes=t * DV * (2 * dg * 4 + dh * 2 + dh * 4) + 2 * nseq * dh * DV * DV * 4)
        qfv = rnd(t, dh * 3 * DV, dtype=torch.float32)
        b2, lo = f32(dh * DV) * 2, f32(dh * DV) * 0.5
        row("like: hgrn2", phase, lambda: hops.hgrn2(qfv, b2, lo, rec, raw, dh, DV, DV, si, split=True), nbytes=t * dh * DV * 16 + 2 * nseq * dh * DV * DV * 4)
        nw, gated = f32(DV), empty(t, dh * DV)
        row("head_rmsnorm * gate", phase, lambda: hops.head_rmsnorm(raw, nw, 1e-6, gated, dh, DV, gate=ud[:, :dh * DV]), nbytes=t * dh * DV * 8)
        row("like: head_rmsnorm", phase, lambda: hops.head_rmsnorm(raw, nw, 1e-6, gated, dh, DV), nbytes=t * dh * DV * 6)
        # experts
        wr, logits = rnd(e, hid), empty(t, e, dtype=torch.float32)
        row("gemm router (fp32 out)", phase, lambda: hops.linear(h, wr, logits, f32_out=True), 2 * t * e * hid, (e + t) * hid * 2 + t * e * 4)
        logits.normal_()
        up, down = rnd(e, ff, hid), rnd(e, hid, ff)
        ws = mops.MoEWorkspace(t, top, e, hid, ff, "cuda", bf)
        fl, by = 4 * t * top * ff * hid, min(e, t * top) * 2 * ff * hid * 2 + t * top * (2 * hid + 2 * ff) * 2
        row("experts: route, permute, gather, up, down", phase, lambda: mops.relu2_experts(h, logits, up, down, ws, top, groups, kept), fl, by)
        half, gu, lg, acc = 128, rnd(e, 2 * ff, hid), logits.to(bf), empty(t, hid)
        fl, by = 6 * t * top * ff * hid, min(e, t * top) * 3 * ff * hid * 2 + t * top * (2 * hid + 2 * ff) * 2
        row("like: experts with a gate, combine", phase, lambda: mops.moe_experts(h, lg, gu, down, ws, acc, top, True, half, accumulate=False), fl, by)
        del up, down, gu, ws
        torch.cuda.empty_cache()
    ops.check_status()
    return rows


def main(sizes, json_path="") -> dict:
    pk, timer = peaks(), Timer()
    doc = {"peaks": pk, "sizes": {}}
    for size in sizes:
        new, like = configs(size)
        prefills, decode = [(1, 4096), (4, 1024)], (64, 2048)
        res = {"dezudra": run_model(new, prefills, decode)}
        torch.cuda.empty_cache()
        res["moe gqa"] = run_model(like, prefills, decode)
        torch.cuda.empty_cache()
        doc["sizes"][size] = {"config": SIZES[size], "weights_gb": {"dezudra": new.weight_bytes() / 1e9, "moe gqa": like.weight_bytes() / 1e9},
                              "throughput": {m: {k: {"ms": round(ms, 3), "tok_s": round(t / ms * 1e3)} for k, (t, ms) in r.items()} for m, r in res.items()},
                              "kernels": kernel_rows(size, timer, pk)}
        print(f"== {size} {SIZES[size]}", file=sys.stderr)
        for m, r in doc["sizes"][size]["throughput"].items():
            for k, v in r.items():
                print(f"  {m:8s} {k:28s} {v['ms']:9.3f} ms {v['tok_s']:>9d} tok/s", file=sys.stderr)
        for r in doc["sizes"][size]["kernels"]:
            print(f"  {r['step']:24s} {r['kernel']:44s} {r['ms']:8.4f} ms  roofline {r['roofline_ms']:8.4f}  {r['of_roofline']:.3f}  "
                  f"{r['TF/s'] or '':>7} TF/s {r['GB/s'] or '':>8} GB/s", file=sys.stderr)
    if json_path:
        with open(json_path, "w", encoding="utf-8") as f:
            json.dump(doc, f, indent=1)
    return doc
