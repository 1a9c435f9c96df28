"""Prefill and decode throughput of decoders with matrix memories and tied-key attention (models/midisun.py) beside a decoder of
delta-rule and differential-attention layers (models/dezudra.py) of equal width, depth, heads, window and expert operations, and the row
of every kernel beside the like kernel of the existing models.  Random weights, synthetic tokens; steps and timing as in
:mod:`.hybrid_bench`.

    python bench.py --hybrid --hybrid-design midisun [--hybrid-sizes small,large] [--hybrid-json out.json]
"""
from __future__ import annotations

import json
import sys

import torch

from .. import ops
from ..models.hybrid import DeltaSpec, DiffSpec, HybridConfig, LayerSpec, MemorySpec, MlpSpec, MoeSpec, TiedSpec, distance_slopes
from ..ops import hybrid as hops
from ..ops import moe as mops
from .delta_bench import visible_pairs
from .hybrid_bench import VOCAB, _plan, run_model
from .kernel_bench import Timer, peaks

# hidden, layers, attention heads / KV heads (of 128), window, retention heads (of 128 x 128), mLSTM heads (of 128 x 256), experts, chosen, groups,
# groups kept, expert feed-forward, dense feed-forward
SIZES = {
    "small": (2048, 12, 16, 4, 1024, 16, 8, 32, 4, 4, 2, 1024, 6144),
    "medium": (3072, 8, 24, 8, 2048, 24, 12, 64, 6, 8, 4, 1024, 9216),
    "large": (4096, 8, 32, 8, 4096, 32, 16, 16, 2, 4, 2, 4096, 14336),
}
D = 128            # attention heads, memory keys, retention values
MV = 256           # mLSTM values
TAPS, GROUPS = 4, 4


def configs(size: str):
    hid, layers, hq, hkv, window, rh, mh, e, top, groups, kept, ff, dense = SIZES[size]
    moe = MoeSpec(e, top, ff, groups, kept, True, "silu", bias=True, score="sigmoid", group_best=2)
    tied = TiedSpec(hq, hkv, D, D ** -0.5, 30.0, window)
    ret = MemorySpec(rh, D, D, decay=tuple(1 - 2.0 ** -(5 + 6 * a / rh) for a in range(rh)), rot_dims=D, rot_base=1e4)
    mem = MemorySpec(mh, D, MV, gate_cap=10.0)
    new = HybridConfig(vocab=VOCAB, hidden=hid, layers=[LayerSpec((tied, ret, ret, mem)[i % 4], MlpSpec(dense, "silu") if i % 4 == 0 else moe) for i in range(layers)],
                       residual="pre", norm_groups=GROUPS, input_taps=TAPS, ff_input_conv=False, residual_gates=True, embed_normed=False, name=f"midisun-{size}")
    # experts there have two matrices: half as many channels again for as many operations
    other = MoeSpec(e, top, ff * 3 // 2, groups, kept)
    diff = DiffSpec(hq, hkv, D // 2, D, TAPS, 0.125, 0.5, window, 0, D // 2, 1e4)
    like = HybridConfig(vocab=VOCAB, hidden=hid, layers=[LayerSpec(diff if i % 4 == 0 else DeltaSpec(rh, rh, D, D, TAPS), other) for i in range(layers)],
                        residual="sandwich", name=f"dezudra-{size}")
    return new, like


def kernel_rows(size: str, timer, pk):
    """One row per kernel: this design's, and behind it the like kernel of the existing models ("like: ...") at the same shapes."""
    hid, _, hq, hkv, window, rh, mh, e, top, groups, kept, ff, _ = SIZES[size]
    bf, f4 = torch.bfloat16, torch.float32
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
        product = lambda n, k, out=2: dict(flops=2 * t * n * k, nbytes=(n + t) * k * 2 + t * n * out)
        # residual, norms, input convolutions, gates
        x, x1, y, h, n1, gate = rnd(t, hid, dtype=f4), rnd(t, hid, dtype=f4), rnd(t, hid), empty(t, hid), empty(t, hid), rnd(t, hid)
        w, one, gb = hops.RmsNorm(f32(hid), 1e-6, GROUPS), hops.RmsNorm(f32(hid), 1e-6), f32(hid)
        conv, state, factor = f32(TAPS, hid), torch.zeros(nseq, TAPS - 1, hid, device="cuda"), empty(t * GROUPS, dtype=f4) if t > 512 else None
        routed = hops.ExpertRows(rnd(t * top, hid), torch.randperm(t * top, device="cuda").int().view(t, top), f32(t, top))
        slots = 2 * nseq * (TAPS - 1) * hid * 4
        row("norm_conv_step (gate, groups, both outputs)", phase,
            lambda: hops.norm_conv_step(x, x1, hops.GatedRows(y, gate, gb), None, w, conv, state, h, si, factor, n1), nbytes=t * hid * (8 + 4 + 4) + slots)
        row("norm_conv_step over expert rows (gate ..)", phase,
            lambda: hops.norm_conv_step(x, x1, hops.GatedRows(routed, gate, gb), None, w, conv, state, h, si, factor, n1), nbytes=t * hid * (8 + 2 + 2 * top + 4) + slots)
        row("like: norm_conv_step", phase, lambda: hops.norm_conv_step(x, x1, y, None, one, conv, state, h, si, factor), nbytes=t * hid * (8 + 2 + 2) + slots)
        row("like: norm_conv_step over expert rows", phase, lambda: hops.norm_conv_step(x, x1, routed, None, one, conv, state, h, si, factor),
            nbytes=t * hid * (8 + 2 * top + 2) + slots)
        row("norm_step (gate, groups, bias)", phase, lambda: hops.norm_step(x, hops.GatedRows(y, gate, gb, gb), None, w, h), nbytes=t * hid * (8 + 4 + 2))
        row("like: norm_step", phase, lambda: hops.norm_step(x, y, None, one, h), nbytes=t * hid * (8 + 2 + 2))
        wg = rnd(hid, hid)
        row("gemm residual gate", phase, lambda: hops.linear(h, wg, gate), **product(hid, hid))
        # attention
        n = (hq + hkv) * D + hq
        wq, u, q, attn = rnd(n, hid), empty(t, (n + 7) // 8 * 8), empty(t, hq * D), empty(t, hq * D)
        row("gemm q|k|gates", phase, lambda: hops.linear(h, wq, u[:, :n]), **product(n, hid))
        wl, qkv = rnd((hq + 2 * hkv) * D, hid), rnd(t, (hq + 2 * hkv) * D)
        row("like: gemm qkv", phase, lambda: ops.gemm(h, wl, out=qkv), **product(wl.shape[0], hid))
        u.normal_()
        pool = rnd(npages, hops.tied_page_elems(hkv, D))
        pool.view(f4)[:, hkv * 16 * D // 2:] = 0.1 / 30
        qb, kb, qg = f32(hq * D), f32(hkv * D), f32(hq * D)
        row("tied_append", phase, lambda: hops.tied_append(u, qb, kb, qg, 1e-6, D ** -0.5 / 30, q, pool, si.slots, hq, hkv, D, D), nbytes=2 * t * (hq + hkv) * D * 2)
        kv = rnd(npages, hkv, 2, 16, D)
        table = ops.reference.rope_table(ctx + 1, D, 1e4, "cuda")
        row("like: rope_kv_append", phase, lambda: ops.rope_kv_append(qkv, si.positions, si.slots, table, kv, hq, hkv, D), nbytes=2 * t * (hq + 2 * hkv) * D * 2)
        q.normal_()
        pairs, keys = visible_pairs(chunks, window, 0)
        fl, by, lby = 4 * pairs * hq * D, keys * hkv * (D * 2 + 4) + 2 * t * hq * D * 2, keys * hkv * 2 * D * 2 + 2 * t * hq * D * 2
        slope, sink, out = distance_slopes(hq, "cuda"), f32(hq), empty(t, hq * D)
        hg = u[:, (hq + hkv) * D:(hq + hkv) * D + hq]
        if prompt:
            row("tied_attention (prompt)", phase, lambda: hops.tied_attention(q, attn, pool, si, hq, hkv, D, D, 30.0, slope, sink, window, hg), fl, by)
            row("  the same without a cap", phase, lambda: hops.tied_attention(q, attn, pool, si, hq, hkv, D, D, 0.0, slope, sink, window, hg), fl, by)
            row("like: paged_prefill (window, tcgen05)", phase, lambda: ops.paged_prefill(qkv, out, kv, si.page_table, si.ctx_len, si.cu_q, si.tile_seq, si.tile_q0,
                                                                                        si.num_tiles, hq, hkv, D, None, window), fl, lby)
        else:
            ctas = hkv * -(-(hq // hkv) // 16)
            splits = 1
            while 2 * splits * ctas * nseq <= 296 and min(ctx, window) // (2 * splits) >= 128:
                splits *= 2
            cnt = torch.zeros(nseq * ctas, dtype=torch.int32, device="cuda")
            po, pm = empty(nseq * ctas * 16 * splits * D, dtype=f4), empty(nseq * ctas * 32 * splits, dtype=f4)
            row(f"tied_attention (decode, {splits} splits)", phase, lambda: hops.tied_attention(q, attn, pool, si, hq, hkv, D, D, 30.0, slope, sink, window, hg, splits, po, pm,
                                                                                               cnt), fl, by)
            row("like: paged_decode (window)", phase, lambda: ops.paged_decode(qkv, out, kv, si.page_table, si.ctx_len, hq, hkv, D, None, 1, None, None, window), fl, lby)
        wo = rnd(hid, hq * D)
        row("gemm o", phase, lambda: hops.linear(attn, wo, y), **product(hid, hq * D))
        # memories
        work: dict = {}

        def scratch(name, shape):
            size = 1
            for s in shape:
                size *= s
            if name not in work or work[name].numel() < size:
                work[name] = empty(size, dtype=f4)
            return work[name][:size].view(shape)

        turns = empty(t, D // 2, 2, dtype=f4)
        freq = torch.rand(D // 2, dtype=torch.float64, device="cuda")
        row("turn_table (once a step)", phase, lambda: hops.turn_table(si.positions, freq, turns), nbytes=t * D * 4)
        dec = torch.linspace(0.96, 0.999, rh, device="cuda")
        dec = torch.stack([dec, dec.log()]).contiguous()
        for what, heads, vd, gated in (("retention", rh, D, False), ("mlstm", mh, MV, True)):
            width = heads * (2 * D + 2 * vd)
            wp, p, raw, o = rnd(width, hid), empty(t, width), empty(t, heads * vd, dtype=f4), empty(t, heads * vd)
            row(f"gemm q|k|v|gate ({what})", phase, lambda: hops.linear(h, wp, p), **product(width, hid))
            p.normal_()
            st, peak = torch.zeros(nseq, heads, vd + gated, D, device="cuda"), torch.zeros(nseq, heads, device="cuda")
            logits = rnd(t, 2 * heads, dtype=f4) if gated else None
            if gated:
                wi = rnd(2 * heads, hid)
                row("gemm input|forget gates (fp32 out)", phase, lambda: hops.linear(h, wi, logits, f32_out=True), **product(2 * heads, hid, 4))
            bias = f32(2 * heads) + 2 if gated else None
            row(f"decay_memory ({what})", phase, lambda: hops.decay_memory(p, None if gated else turns, logits, bias, 10.0, None if gated else dec, st, peak if gated else None,
                                                                          raw, heads, D, vd, 1.0, 1.0, si, blocks=True, scratch=scratch),
                nbytes=t * heads * ((2 * D + vd) * 2 + vd * 4) + 2 * nseq * heads * (vd + gated) * D * 4)
            nw = f32(heads * vd)
            row(f"head_rmsnorm * gate ({what})", phase, lambda: hops.head_rmsnorm(raw, nw if gated else None, 1e-6, o, heads, vd, gate=p[:, heads * (2 * D + vd):],
                                                                                 gate_act="sigmoid" if gated else "silu"), nbytes=t * heads * vd * 8)
            wd = rnd(hid, heads * vd)
            row(f"gemm o ({what})", phase, lambda: hops.linear(o, wd, y), **product(hid, heads * vd))
        rec, raw, o = torch.zeros(nseq, rh, D, D, device="cuda"), empty(t, rh * D, dtype=f4), empty(t, rh * D)
        qfv = rnd(t, rh * 3 * D, dtype=f4)
        b2, lo = f32(rh * D) * 2, f32(rh * D) * 0.5
        row("like: hgrn2", phase, lambda: hops.hgrn2(qfv, b2, lo, rec, raw, rh, D, D, si, split=True, scratch=scratch), nbytes=t * rh * D * 16 + 2 * nseq * rh * D * D * 4)
        qk, v, gates = rnd(t, 2 * rh * D, dtype=f4), rnd(t, rh * D), -f32(t, rh, 2)
        row("like: delta_rule", phase, lambda: hops.delta_rule(qk, v, gates, rec, raw, rh, rh, D, D, si, blocks=True, scratch=scratch),
            nbytes=t * D * (2 * rh * 4 + rh * 2 + rh * 4) + 2 * nseq * rh * D * D * 4)
        row("like: head_rmsnorm * gate", phase, lambda: hops.head_rmsnorm(raw, b2[:D], 1e-6, o, rh, D, gate=v), nbytes=t * rh * D * 8)
        # experts
        wr, logits, corr = rnd(e, hid), empty(t, e, dtype=f4), f32(e)
        row("gemm router (fp32 out)", phase, lambda: hops.linear(h, wr, logits, f32_out=True), **product(e, hid, 4))
        logits.normal_()
        half, gu, down, lg, acc = 128, rnd(e, 2 * ff, hid), rnd(e, hid, ff), logits.to(bf), empty(t, hid)
        corr *= 0.01                                      # choices stay spread over the experts
        ws = mops.MoEWorkspace(t, top, e, hid, ff, "cuda", bf)
        fl, by = 6 * t * top * ff * hid, min(e, t * top) * 3 * ff * hid * 2 + t * top * (2 * hid + 2 * ff) * 2
        row("experts: route, permute, gather, up, down", phase,
            lambda: mops.routed_experts(h, logits, gu, down, ws, top, "silu", half, groups, kept, True, corr, "sigmoid", 2), fl, by)
        row("like: experts with a gate, combine", phase, lambda: mops.moe_experts(h, lg, gu, down, ws, acc, top, True, half, accumulate=False), fl, by)
        del gu, down, ws, work
        torch.cuda.empty_cache()
    ops.check_status()
    return rows


def main(sizes, json_path="") -> dict:
    pk, timer = peaks(), Timer()
    doc = {"peaks": pk, "sizes": {}}
    for size in sizes:
        new, like = configs(size)
        prefills, decode = [(1, 4096), (4, 1024)], (64, 2048)
        res = {"midisun": run_model(new, prefills, decode)}
        torch.cuda.empty_cache()
        res["dezudra"] = run_model(like, prefills, decode)
        torch.cuda.empty_cache()
        doc["sizes"][size] = {"config": SIZES[size], "weights_gb": {"midisun": new.weight_bytes() / 1e9, "dezudra": like.weight_bytes() / 1e9},
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
