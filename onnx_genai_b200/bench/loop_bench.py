"""Prefill and decode throughput of looped latent-attention decoders (models/fizesun.py) beside a Rilelorn decoder of latent layers with
equal width, layer runs, heads, latents and multiply-adds per token, and the row of every kernel beside the like kernel of the
existing models.  Random weights, synthetic tokens; steps and timing as in :mod:`.hybrid_bench`.

    python bench.py --hybrid --hybrid-design fizesun [--hybrid-sizes small,large] [--hybrid-json out.json]
"""
from __future__ import annotations

import json
import sys

import torch

from .. import ops
from ..models import hybrid as models
from ..models.hybrid import HybridConfig, LatentSpec, LayerSpec, LoopSpec, MlpSpec, MoeSpec
from ..ops import hybrid as hops
from ..ops import moe as mops
from .hybrid_bench import VOCAB, _plan, run_model, seen_pairs
from .kernel_bench import Timer, peaks

# hidden, layers, loop (start, stop, times), heads, dim, rotated, value width, latent, dense feed-forward, experts, chosen, expert feed-forward.
# A shared expert of the same size runs beside the chosen ones; dense and expert layers alternate and cost the same per token.
SIZES = {
    "small": (2048, 8, (2, 6, 2), 16, 64, 32, 64, 256, 6144, 32, 3, 1024),
    "medium": (3072, 6, (1, 4, 2), 24, 128, 64, 128, 512, 9216, 64, 5, 1024),
    "large": (4096, 4, (0, 2, 2), 32, 128, 64, 128, 512, 12288, 32, 3, 2048),
}
TAPS = 4
LIMIT = 7.0


def configs(size: str):
    hid, layers, loop, heads, d, r, v, rank, ff, e, top, fe = SIZES[size]
    latent = LatentSpec(heads, d, v, rank, (d + r) ** -0.5, rot_dim=r, rot_base=5e4, gated=True)
    moe = MoeSpec(e, top, fe, renormalize=True, act="clamp_glu", limit=LIMIT, shared_inter=fe, shared_limit=LIMIT, bias=True)
    specs = [LayerSpec(latent, moe if i % 2 else MlpSpec(ff, "xielu")) for i in range(layers)]
    new = HybridConfig(vocab=VOCAB, hidden=hid, layers=specs, residual="pre", input_taps=TAPS, loop=LoopSpec(*loop), name=f"fizesun-{size}")
    like = HybridConfig(vocab=VOCAB, hidden=hid, streams=2, name=f"latent-{size}",
                        layers=[LayerSpec(LatentSpec(heads, v, v, rank, v ** -0.5), MlpSpec(ff * 2 // 3)) for _ in new.runs])
    return new, like


def kernel_rows(size: str, timer, pk):
    """One row per kernel: this design's, and behind it the like kernel of the existing models ("like: ...") at the same shapes."""
    hid, _, _, heads, d, r, dv, rank, ff, e, top, fe = SIZES[size]
    bf = torch.bfloat16
    m = LatentSpec(heads, d, dv, rank, (d + r) ** -0.5, rot_dim=r, gated=True)
    plain = LatentSpec(heads, dv, dv, rank, dv ** -0.5)
    qw, kw = m.q_width, m.key_width
    rnd = lambda *s, dtype=bf: (torch.randn(*s, device="cuda") * 0.1).to(dtype)
    f32 = lambda *s: torch.rand(*s, device="cuda")
    empty = lambda *s, dtype=bf: torch.empty(*s, dtype=dtype, device="cuda")
    i32 = lambda *s: torch.zeros(*s, dtype=torch.int32, device="cuda")
    rows = []

    def row(name, phase, fn, flops=0, nbytes=0):
        ms, _ = timer.time(fn)
        bound = max(flops / (pk["bf16_tflops"] * 1e12), nbytes / (pk["hbm_gbs"] * 1e9)) * 1e3
        rows.append({"kernel": name, "step": phase, "ms": round(ms, 4), "roofline_ms": round(bound, 4), "of_roofline": round(bound / ms, 3),
                     "TF/s": round(flops / ms / 1e9, 1) if flops else None, "GB/s": round(nbytes / ms / 1e6, 1) if nbytes else None})

    for phase, parts in (("prefill 4096", [(0, 4096)]), ("prefill 4x1024", [(0, 1024)] * 4), ("decode 64", [(2047, 1)] * 64),
                         ("decode 64, context 8192", [(8191, 1)] * 64)):
        t, nseq = sum(n for _, n in parts), len(parts)
        ctx = max(a + n for a, n in parts)
        mp, npages = (ctx + 15) // 16, sum((a + n + 15) // 16 for a, n in parts)
        si = _plan(parts, mp, npages)
        prompt = si.num_prefill_seqs > 0
        # residual, norms, input convolutions
        x0, x1, y, h = rnd(t, hid, dtype=torch.float32), empty(t, hid, dtype=torch.float32), rnd(t, hid), empty(t, hid)
        w = hops.RmsNorm(f32(hid), 1e-6)
        conv, state = f32(TAPS, hid), torch.zeros(nseq, TAPS - 1, hid, device="cuda")
        sb = 2 * nseq * (TAPS - 1) * hid * 4
        factor = f32(t) if prompt else None
        row("norm_conv_step", phase, lambda: hops.norm_conv_step(x0, x1, y, None, w, conv, state, h, si, factor), nbytes=t * hid * (8 + 4) + sb)
        routed = hops.ExpertRows(rnd(t * top, hid), torch.randperm(t * top, device="cuda").int().view(t, top), f32(t, top), rnd(t, hid), f32(t, e + 8)[:, e])
        row("norm_conv_step over expert rows", phase, lambda: hops.norm_conv_step(x0, x1, routed, None, w, conv, state, h, si, factor),
            nbytes=t * hid * (8 + 2 + 2 * (top + 1)) + sb)
        xs0, xs1, prev, amount = rnd(t, 2, hid, dtype=torch.float32), empty(t, 2, hid, dtype=torch.float32), f32(nseq, hid), f32(hid)
        hc, dyn = hops.HyperConnection(f32(2), f32(2), f32(2, 2)), hops.DynamicTanh(f32(1), f32(hid), f32(hid))
        row("like: hyper_step + shift", phase, lambda: hops.hyper_step(xs0, xs1, y, hc, hc.read, dyn, h, si, shift=amount, prev=prev),
            nbytes=t * hid * (16 + 4) + 2 * nseq * hid * 4)
        row("like: norm_step over expert rows", phase, lambda: hops.norm_step(x0, hops.ExpertRows(routed.rows, routed.pos, routed.weight), w, w, h),
            nbytes=t * hid * (8 + 2 + 2 * top))
        del xs0, xs1
        # entering a pass
        both, wl = rnd(t, 2 * hid), rnd(hid, 2 * hid)
        row("norm_step, copy beside the embedding", phase, lambda: hops.norm_step(x0, y, None, None, both[:, :hid]), nbytes=t * hid * 12)
        row("gemm pass (fp32 out)", phase, lambda: hops.linear(both, wl, x1, f32_out=True), 4 * t * hid * hid, 2 * hid * (2 * t + 2 * hid) + t * hid * 4)
        del both, wl
        # latent attention
        wq, qc = rnd(m.proj_width, hid), empty(t, models.pad8(m.proj_width))
        row("gemm q|latent|rotated|gates", phase, lambda: hops.linear(h, wq, qc[:, :m.proj_width]), 2 * t * m.proj_width * hid,
            (m.proj_width + t) * hid * 2 + t * m.proj_width * 2)
        wp, qp = rnd(plain.proj_width, hid), empty(t, plain.proj_width)
        row("like: gemm q|latent", phase, lambda: hops.linear(h, wp, qp), 2 * t * plain.proj_width * hid, (plain.proj_width + t) * hid * 2 + t * plain.proj_width * 2)
        qc.normal_()
        pool, pool1, cn = rnd(npages, 16, kw), rnd(npages, 16, rank), f32(rank)
        qa, oc = rnd(t * heads, kw), empty(t * heads, rank)
        rope = hops.LatentRope(models.rotation(r, 5e4, "cuda"), si.positions, heads, d, qa, rank, t)
        row("latent_append + rotations", phase, lambda: hops.latent_append(qc, m.latent_col, cn, 1e-6, si.slots, pool, rank, rope),
            nbytes=2 * t * (kw + heads * r) * 2)
        row("like: latent_append", phase, lambda: hops.latent_append(qp, plain.latent_col, cn, 1e-6, si.slots, pool1, rank), nbytes=2 * t * rank * 2)
        qkv, kv = rnd(t, (heads + 2 * (heads // 4)) * 128), rnd(npages, heads // 4, 2, 16, 128)
        rt = ops.reference.rope_table(ctx + 1, 128, 1e4, "cuda")
        row("like: rope_kv_append (GQA)", phase, lambda: ops.rope_kv_append(qkv, si.positions, si.slots, rt, kv, heads, heads // 4, 128),
            nbytes=2 * t * qkv.shape[1] * 2)
        del qkv, kv
        uk, uv, attn, wb = rnd(heads * rank, d), rnd(heads * dv, rank), empty(t, heads * dv), heads * rank * 2
        row("gemm per head (W_uk^T q)", phase, lambda: hops.linear_batched(qc, uk, qa.view(t, -1), heads, qw, kw), 2 * t * heads * d * rank,
            t * heads * (d + rank) * 2 + wb * d)
        row("gemm per head (W_uv o)", phase, lambda: hops.linear_batched(oc.view(t, -1), uv, attn, heads, rank, dv), 2 * t * heads * dv * rank,
            t * heads * (dv + rank) * 2 + wb * dv)
        uk1, qa1 = rnd(heads * rank, dv), empty(t, heads * rank)
        row("like: gemm per head (W_uk^T q)", phase, lambda: hops.linear_batched(qp, uk1, qa1, heads, dv, rank), 2 * t * heads * dv * rank,
            t * heads * (dv + rank) * 2 + wb * dv)
        del uk1, qa1
        gate = qc[:, m.gate_col:m.gate_col + heads]
        pairs, keys = seen_pairs(parts, 0), sum(a + n for a, n in parts)
        qa1 = rnd(t * heads, rank)
        if prompt:
            fl = 2 * pairs * heads * (qw + dv)
            row("latent_attention (prompt on the latents)", phase, lambda: hops.latent_attention(qa, oc, pool, si, heads, kw, 0.1, 0, vrank=rank, gate=gate),
                2 * pairs * heads * (kw + rank), keys * kw * 2 + t * heads * (kw + rank) * 2)
            row("like: latent_attention (prompt on the latents)", phase, lambda: hops.latent_attention(qa1, oc, pool1, si, heads, rank, 0.1, 0),
                4 * pairs * heads * rank, keys * rank * 2 + 2 * t * heads * rank * 2)
            n = hops.visible_pages(si, 0)
            for name, s, pl, q, g in (("latent prompt, expanded K/V (3 kernels)", m, pool, qc, gate), ("like: latent prompt, expanded K/V (3 kernels)", plain, pool1, qp, None)):
                kc, vc = models.chunks(s.q_width), models.chunks(s.vdim)
                dense, kvp, table, kvw = empty(n * 16, s.key_width), empty(n, heads, kc + vc, 16, 64), i32(nseq, mp), rnd(heads * (kc + vc) * 64, s.key_width)
                row(name, phase, lambda: hops.latent_prefill_expanded(q, attn, pl, kvw, si, heads, kc, vc, s.q_width, s.vdim, 0.1, 0, n, dense, kvp, table, g),
                    2 * pairs * heads * (s.q_width + s.vdim) + 2 * n * 16 * rank * heads * (s.dim + s.vdim), keys * s.key_width * 2 + t * heads * (s.q_width + s.vdim) * 2)
            del dense, kvp, kvw
        else:
            per = -(-heads // 32) * nseq
            for name, q, pl, width, g in (("latent_attention", qa, pool, kw, gate), ("like: latent_attention", qa1, pool1, rank, None)):
                splits = 1
                while 2 * splits * per <= 148 * (2 if width <= 128 else 1) and ctx // (2 * splits) >= 128:
                    splits *= 2
                cnt, po, pm = i32(4096), empty(t * heads * splits * rank, dtype=torch.float32), empty(t * heads * splits * 2, dtype=torch.float32)
                row(f"{name} (decode, {splits} splits)", phase, lambda: hops.latent_attention(q, oc, pl, si, heads, width, 0.1, 0, splits, po, pm, cnt, vrank=rank, gate=g),
                    2 * pairs * heads * (width + rank), keys * width * 2 + t * heads * (width + rank) * 2)
        wo = rnd(hid, heads * dv)
        row("gemm o", phase, lambda: hops.linear(attn, wo, y), 2 * t * hid * heads * dv, (hid + t) * heads * dv * 2 + t * hid * 2)
        del qa, qa1, oc, pool, pool1, uk, uv, wo, wq, wp
        # feed-forwards
        up, mid, down = rnd(ff, hid), empty(t, ff), rnd(hid, ff)
        fl, by = 2 * t * ff * hid, (ff + t) * hid * 2 + t * ff * 2
        row("gemm up (xIELU)", phase, lambda: hops.act_linear(h, up, models.xielu(0.3, -0.2), mid), fl, by)
        row("gemm down", phase, lambda: hops.linear(mid, down, y), fl, by)
        gu, act = rnd(ff * 4 // 3, hid), empty(t, ff * 2 // 3)
        row("like: gemm gate_up (gelu gate)", phase, lambda: hops.gated_linear(h, gu, 128, "gelu_tanh", act), 4 * t * act.shape[1] * hid,
            (gu.shape[0] + t) * hid * 2 + t * act.shape[1] * 2)
        del up, mid, down, gu, act
        wr, logits = rnd(e + 1, hid), empty(t, models.pad8(e + 1), dtype=torch.float32)
        row("gemm router|shared gate (fp32 out)", phase, lambda: hops.linear(h, wr, logits[:, :e + 1], f32_out=True), 2 * t * (e + 1) * hid,
            (e + 1 + t) * hid * 2 + t * (e + 1) * 4)
        row("like: gemm router", phase, lambda: hops.linear(h, wr[:e], logits[:, :e], f32_out=True), 2 * t * e * hid, (e + t) * hid * 2 + t * e * 4)
        logits.normal_()
        gu, dn, bias = rnd(e, 2 * fe, hid), rnd(e, hid, fe), f32(e)
        ws = mops.MoEWorkspace(t, top, e, hid, fe, "cuda", bf)
        fl, by = 6 * t * top * fe * hid, min(e, t * top) * 3 * fe * hid * 2 + t * top * (2 * hid + 2 * fe) * 2
        glu = hops.Act("clamp_glu", LIMIT)
        row("experts: route, permute, gather, gate_up, down", phase, lambda: mops.routed_experts(h, logits[:, :e], gu, dn, ws, top, glu, 128, renormalize=True, bias=bias), fl, by)
        lg, acc = logits[:, :e].to(bf), empty(t, hid)
        row("like: experts (silu gate), combine", phase, lambda: mops.moe_experts(h, lg, gu, dn, ws, acc, top, True, 128, accumulate=False), fl, by)
        sg, sd, mid = rnd(2 * fe, hid), rnd(hid, fe), empty(t, fe)
        fl, by = 4 * t * fe * hid, (2 * fe + t) * hid * 2 + t * fe * 2
        row("shared expert gemm gate_up (clamped gate)", phase, lambda: hops.gated_linear(h, sg, 128, glu, mid), fl, by)
        row("like: gemm gate_up (gelu gate), same size", phase, lambda: hops.gated_linear(h, sg, 128, "gelu_tanh", mid), fl, by)
        row("shared expert gemm down", phase, lambda: hops.linear(mid, sd, y), 2 * t * fe * hid, (fe + t) * hid * 2 + t * fe * 2)
        del gu, dn, ws, sg, sd
        torch.cuda.empty_cache()
    ops.check_status()
    return rows


def main(sizes, json_path="") -> dict:
    pk, timer = peaks(), Timer()
    doc = {"peaks": pk, "sizes": {}}
    for size in sizes:
        new, like = configs(size)
        prefills, decode = [(1, 4096), (4, 1024)], (64, 2048)
        res = {"fizesun": run_model(new, prefills, decode)}
        torch.cuda.empty_cache()
        res["latent"] = run_model(like, prefills, decode)
        torch.cuda.empty_cache()
        doc["sizes"][size] = {"config": SIZES[size], "weights_gb": {"fizesun": new.weight_bytes() / 1e9, "latent": like.weight_bytes() / 1e9},
                              "throughput": {m: {k: {"ms": round(ms, 3), "tok_s": round(t / ms * 1e3)} for k, (t, ms) in r.items()} for m, r in res.items()},
                              "kernels": kernel_rows(size, timer, pk)}
        print(f"== {size} {SIZES[size]}", file=sys.stderr)
        for m, r in doc["sizes"][size]["throughput"].items():
            for k, v in r.items():
                print(f"  {m:8s} {k:28s} {v['ms']:9.3f} ms {v['tok_s']:>9d} tok/s", file=sys.stderr)
        for r in doc["sizes"][size]["kernels"]:
            print(f"  {r['step']:24s} {r['kernel']:48s} {r['ms']:8.4f} ms  roofline {r['roofline_ms']:8.4f}  {r['of_roofline']:.3f}  "
                  f"{r['TF/s'] or '':>7} TF/s {r['GB/s'] or '':>8} GB/s", file=sys.stderr)
    if json_path:
        with open(json_path, "w", encoding="utf-8") as f:
            json.dump(doc, f, indent=1)
    return doc
