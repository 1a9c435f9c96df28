"""Plain PyTorch fp32 statements of every fused op.

These are the numerics oracle for the CUDA kernels (tests compare each kernel against the
function of the same name here) and the execution path for CPU tensors.  Conventions follow the
reference's CPU kernels: RMSNorm with fp32 statistics, half-rotation or interleaved rotary
(crates/onnx-runtime-ep-cuda/src/kernels/rotary_embedding.rs:45), GQA causal softmax
(crates/onnx-runtime-ep-cpu/src/kernels/group_query_attention.rs), MatMulNBits dequantisation
``(code - zp) * scale`` with the low nibble holding the even k
(crates/onnx-runtime-ep-cpu/src/kernels/matmul_nbits.rs:1-17), sampler order temperature ->
top-k -> top-p -> min-p (crates/onnx-genai-engine/src/processors.rs:18-215) and argmax ties to
the lowest token id (crates/onnx-genai-engine/src/sampling.rs:120-132).
"""
from __future__ import annotations

import math

import torch

PAGE = 16


def gemm(a, w, bias=None, residual=None, epilogue="none", out_dtype=None):
    """a [M,K] @ w[N,K]^T with fp32 accumulation.  ``swiglu``: w rows are tile-interleaved gate|up."""
    y = a.float() @ w.float().t()
    if bias is not None:
        y = y + bias.float()
    if epilogue == "residual":
        y = y + residual.float()
    out_dtype = out_dtype or a.dtype
    return y.to(out_dtype)


def swiglu_packed(a, w_packed, half, out_dtype=None):
    """SwiGLU over a weight packed by :func:`pack_gate_up` with tile half-width ``half``."""
    y = a.float() @ w_packed.float().t()
    m, n = y.shape
    y = y.view(m, n // (2 * half), 2, half)
    g, u = y[:, :, 0, :], y[:, :, 1, :]
    return (torch.nn.functional.silu(g) * u).reshape(m, n // 2).to(out_dtype or a.dtype)


def pack_gate_up(gate_w, up_w, half):
    """Interleave gate and up projection rows in blocks of ``half`` so one GEMM tile of width
    ``2*half`` holds matching gate and up columns: [g0..g(half-1), u0..u(half-1), g(half).. ...]."""
    inter, k = gate_w.shape
    assert inter % half == 0, (inter, half)
    g = gate_w.view(inter // half, 1, half, k)
    u = up_w.view(inter // half, 1, half, k)
    return torch.cat([g, u], dim=1).reshape(2 * inter, k).contiguous()


def rmsnorm(x, weight, eps, delta=None):
    """Returns (normed, new_residual).  With ``delta`` the residual is x + delta, rounded to x.dtype first."""
    if delta is not None:
        x = (x.float() + delta.float()).to(x.dtype)
    xf = x.float()
    inv = torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    return (xf * inv * weight.float()).to(x.dtype), x


def silu_mul(gate_up):
    inter = gate_up.shape[-1] // 2
    g, u = gate_up[..., :inter].float(), gate_up[..., inter:].float()
    return (torch.nn.functional.silu(g) * u).to(gate_up.dtype)


def rope_table(max_pos, rotary_dim, theta, device="cpu"):
    """[max_pos, rotary_dim/2, 2] fp32 (cos, sin), computed in float64 then rounded."""
    half = rotary_dim // 2
    inv_freq = 1.0 / (theta ** (torch.arange(0, half, dtype=torch.float64) * 2.0 / rotary_dim))
    ang = torch.arange(max_pos, dtype=torch.float64)[:, None] * inv_freq[None, :]
    return torch.stack([ang.cos(), ang.sin()], dim=-1).float().to(device)


def apply_rope(x, positions, cos_sin, rotary_dim, interleaved=False):
    """x [T, H, D] -> rotated copy (fp32 math, result in x.dtype)."""
    t, h, d = x.shape
    half = rotary_dim // 2
    cs = cos_sin[positions.long()]  # [T, half, 2]
    c, s = cs[..., 0][:, None, :], cs[..., 1][:, None, :]
    xf = x.float().clone()
    if interleaved:
        x0, x1 = xf[..., 0:rotary_dim:2], xf[..., 1:rotary_dim:2]
        r0, r1 = x0 * c - x1 * s, x1 * c + x0 * s
        xf[..., 0:rotary_dim:2], xf[..., 1:rotary_dim:2] = r0, r1
    else:
        x0, x1 = xf[..., :half], xf[..., half:rotary_dim]
        r0, r1 = x0 * c - x1 * s, x1 * c + x0 * s
        xf[..., :half], xf[..., half:rotary_dim] = r0, r1
    return xf.to(x.dtype)


def e4m3_bytes(x):
    """fp32 -> e4m3 bytes with saturation at +-448 (round to nearest even), as the device conversion does."""
    return x.float().clamp(-448.0, 448.0).to(torch.float8_e4m3fn).view(torch.uint8)


def e5m2_bytes(x):
    """fp32 -> e5m2 with saturation at +-57344 (round to nearest even)."""
    return x.float().clamp(-57344.0, 57344.0).to(torch.float8_e5m2)


def int8_bytes(x):
    """fp32 -> symmetric int8 with saturation at +-127 (round to nearest even)."""
    return torch.round(x.float().clamp(-127.0, 127.0)).to(torch.int8)


def kv_append_fp8(qkv, slots, pool, scales, hq, hkv, d):
    """One-byte page codec (e4m3 in a uint8 pool, symmetric int8 in an int8 pool): one scale per (page, head, K|V),
    fixed by the page's first token at amax * 2 / qmax, qmax = 448 or 127 (headroom
    for the 15 tokens that follow, which saturate to it).  Tokens are taken in row order, so a chunk that starts a
    page and continues it in the same call behaves like one append per token.  pool [P,hkv,2,PAGE,d] uint8,
    scales [P,hkv,2] fp32; qkv already rotated."""
    t = qkv.shape[0]
    v = qkv.view(t, hq + 2 * hkv, d).float()
    qmax, encode = (127.0, int8_bytes) if pool.dtype == torch.int8 else ((57344.0, e5m2_bytes) if pool.dtype == torch.float8_e5m2 else (448.0, e4m3_bytes))
    for i in range(t):
        slot = int(slots[i])
        if slot < 0:
            continue
        page, off = slot // PAGE, slot % PAGE
        for kv in range(2):
            for h in range(hkv):
                vec = v[i, hq + kv * hkv + h]
                if off == 0 or not float(scales[page, h, kv]) > 0.0:
                    scales[page, h, kv] = max(float(vec.abs().max()) * 2.0, 1e-6) / qmax
                inv = torch.tensor(1.0, dtype=torch.float32) / scales[page, h, kv].float()
                pool[page, h, kv, off] = encode(vec * inv)


def rope_kv_append(qkv, positions, slots, cos_sin, pool, hq, hkv, d, rotary_dim=None, interleaved=False, kv_scales=None):
    """In place: rotate q,k inside qkv [T,(hq+2hkv)*d]; write k,v to pool [P,hkv,2,PAGE,d] at slots
    (e4m3 bytes with per-(page, head) scales when ``kv_scales`` is given)."""
    rotary_dim = rotary_dim or d
    t = qkv.shape[0]
    v = qkv.view(t, hq + 2 * hkv, d)
    v[:, : hq + hkv] = apply_rope(v[:, : hq + hkv], positions, cos_sin, rotary_dim, interleaved)
    if kv_scales is not None:
        kv_append_fp8(qkv, slots, pool, kv_scales, hq, hkv, d)
        return qkv
    ok = slots >= 0
    page, off = (slots // PAGE).long(), (slots % PAGE).long()
    k, vv = v[:, hq : hq + hkv], v[:, hq + hkv :]
    pool[page[ok], :, 0, off[ok]] = k[ok].to(pool.dtype)
    pool[page[ok], :, 1, off[ok]] = vv[ok].to(pool.dtype)
    return qkv


def _live_pages(table, n_pages):
    """Page ids of a sequence; entries of released pages (-1: between the attention sinks and the sliding window, never
    visible to a query) are replaced by a live page so that the gather stays in range -- their keys are masked."""
    idx = table[:n_pages].long()
    if bool((idx < 0).any()):
        idx = torch.where(idx < 0, idx[idx >= 0][-1], idx)
    return idx


def _gather_kv(pool, table, ctx):
    n_pages = (ctx + PAGE - 1) // PAGE
    pages = pool[_live_pages(table, n_pages)]  # [n, hkv, 2, PAGE, d]
    k = pages[:, :, 0].permute(1, 0, 2, 3).reshape(pool.shape[1], -1, pool.shape[-1])[:, :ctx]
    v = pages[:, :, 1].permute(1, 0, 2, 3).reshape(pool.shape[1], -1, pool.shape[-1])[:, :ctx]
    return k.float(), v.float()


def paged_attention(q, pool, page_table, ctx_len, cu_q, hq, hkv, d, scale=None, window=0, kv_scales=None, sink=0):
    """Varlen causal GQA over paged KV.  q [T, >=hq*d] (first hq*d columns used); returns [T, hq*d].

    Sequence s owns query rows cu_q[s]:cu_q[s+1]; its last row sits at position ctx_len[s]-1.
    ``kv_scales`` [P,hkv,2] dequantises fp8 pages.  ``window`` > 0 keeps the last ``window`` keys of each query and,
    with ``sink`` > 0, the first ``sink`` keys of the sequence as well (attention sinks).
    """
    scale = scale or 1.0 / math.sqrt(d)
    t = q.shape[0]
    out = torch.zeros(t, hq * d, dtype=q.dtype, device=q.device)
    g = hq // hkv
    for s in range(len(ctx_len)):
        b, e = int(cu_q[s]), int(cu_q[s + 1])
        ctx = int(ctx_len[s])
        if e <= b or ctx <= 0:
            continue
        if kv_scales is not None:
            n_pages = (ctx + PAGE - 1) // PAGE
            idx = _live_pages(page_table[s], n_pages)
            raw = pool[idx]
            if raw.dtype == torch.uint8:   # e4m3 bytes
                raw = raw.view(torch.float8_e4m3fn)
            pages = raw.float() * kv_scales[idx][:, :, :, None, None]
            k = pages[:, :, 0].permute(1, 0, 2, 3).reshape(hkv, -1, d)[:, :ctx]
            v = pages[:, :, 1].permute(1, 0, 2, 3).reshape(hkv, -1, d)[:, :ctx]
        else:
            k, v = _gather_kv(pool, page_table[s], ctx)
        qs = q[b:e, : hq * d].float().view(e - b, hkv, g, d)
        scores = torch.einsum("thgd,hkd->thgk", qs, k) * scale
        qpos = torch.arange(ctx - (e - b), ctx, device=q.device)[:, None]
        kpos = torch.arange(ctx, device=q.device)[None, :]
        mask = kpos <= qpos
        if window > 0:
            mask &= (kpos > qpos - window) | (kpos < sink)
        scores = scores.masked_fill(~mask[:, None, None, :], float("-inf"))
        p = torch.softmax(scores, dim=-1)
        o = torch.einsum("thgk,hkd->thgd", p, v)
        out[b:e] = o.reshape(e - b, hq * d).to(q.dtype)
    return out


def argmax(logits):
    """Lowest index wins ties; NaN never wins."""
    l = logits.float()
    l = torch.where(torch.isnan(l), torch.full_like(l, float("-inf")), l)
    mx = l.max(dim=-1, keepdim=True).values
    idx = torch.arange(l.shape[-1], device=l.device).expand_as(l)
    cand = torch.where(l == mx, idx, torch.full_like(idx, l.shape[-1]))
    return cand.min(dim=-1).values.to(torch.int32)


def sample_weights(logits_row, temperature):
    """Fixed-point weights w = min(round(exp((l - max)/T) * 2^30), 2^30 - 1) as int64 (the device sampler's mass unit)."""
    l = logits_row.float()
    e = torch.exp((l - l.max()) / temperature)
    e = torch.where(torch.isnan(e), torch.zeros_like(e), e)
    return torch.floor(e.double() * 1073741824.0 + 0.5).clamp_max(1073741823.0).to(torch.int64)


def sample_threshold(w, top_k, top_p, min_p):
    """Weight threshold that top-k, then top-p, then min-p leave: a token survives iff its weight is >= the result."""
    vocab = w.numel()
    thr = 1
    total = int(w.sum())
    if 0 < top_k < vocab:
        kth = int(torch.sort(w, descending=True).values[top_k - 1])
        thr = max(thr, kth)
        total = int(w[w >= thr].sum())
    if 0.0 < top_p < 1.0:
        target = max(1, int(float(total) * float(top_p)))
        vals = torch.sort(w[w >= thr], descending=True).values
        csum = torch.cumsum(vals, 0)
        pos = int(torch.searchsorted(csum, torch.tensor(target, dtype=csum.dtype), right=False))
        pos = min(pos, vals.numel() - 1)
        thr = max(thr, int(vals[pos]))
    if min_p > 0.0:
        thr = max(thr, int(torch.tensor(min(min_p, 1.0), dtype=torch.float32) * 1073741824.0))
    return thr


def sample_draw_target(kept, u):
    """(target mass, total mass) of the draw ``u`` over the surviving weights ``kept``."""
    final_total = int(kept.sum())
    uu = min(max(float(torch.tensor(u, dtype=torch.float32)), 0.0), 0.99999994)
    return min(int(uu * float(final_total)), final_total - 1), final_total


def sample_from_weights(w, top_k, top_p, min_p, u):
    """Exact integer statement of the sampler: thresholds keep ties; draw walks tokens in index order."""
    thr = sample_threshold(w, top_k, top_p, min_p)
    kept = torch.where(w >= thr, w, torch.zeros_like(w))
    if int(kept.sum()) == 0:
        return int(torch.argmax(w))
    target, _ = sample_draw_target(kept, u)
    csum = torch.cumsum(kept, 0)
    return int(torch.searchsorted(csum, torch.tensor(target, dtype=csum.dtype), right=True))


def sample(logits, temperature, top_k, top_p, min_p, uniform):
    rows = logits.shape[0]
    out = torch.zeros(rows, dtype=torch.int32)
    for r in range(rows):
        t = float(temperature[r])
        if not t > 0.0:
            out[r] = int(argmax(logits[r : r + 1])[0])
            continue
        w = sample_weights(logits[r].cpu(), t)
        out[r] = sample_from_weights(w, int(top_k[r]), float(top_p[r]), float(min_p[r]), float(uniform[r]))
    return out.to(logits.device)


def spec_verify_greedy(logits, draft, k):
    """logits [S*(k+1), V]; draft [S, k] -> (accept_len [S], out_tokens [S, k+1] padded with -1)."""
    s = draft.shape[0]
    best = argmax(logits).view(s, k + 1)
    accept = torch.zeros(s, dtype=torch.int32)
    out = torch.full((s, k + 1), -1, dtype=torch.int32)
    for i in range(s):
        a = 0
        while a < k and int(draft[i, a]) == int(best[i, a]):
            a += 1
        accept[i] = a
        out[i, :a] = draft[i, :a].to(torch.int32)
        out[i, a] = best[i, a]
    return accept.to(logits.device), out.to(logits.device)


def dequant_w4(qweight, scales, zero_points=None, block=32, k=None):
    """MatMulNBits int4: qweight [N, ceil(K/block), block/2] uint8, scales [N, ceil(K/block)] -> W [N, K] fp32."""
    n, kb, _ = qweight.shape
    lo = (qweight & 0xF).to(torch.int16)
    hi = (qweight >> 4).to(torch.int16)
    codes = torch.stack([lo, hi], dim=-1).reshape(n, kb, block).float()
    if zero_points is None:
        zp = torch.full((n, kb), 8.0, device=qweight.device)
    else:
        zlo = (zero_points & 0xF).to(torch.int16)
        zhi = (zero_points >> 4).to(torch.int16)
        zp = torch.stack([zlo, zhi], dim=-1).reshape(n, -1)[:, :kb].float()
    w = ((codes - zp[:, :, None]) * scales.float()[:, :, None]).reshape(n, kb * block)
    return w[:, :k].contiguous() if k is not None and k < kb * block else w


def quantize_w4(w, block=32, symmetric=True):
    """Block-wise int4 quantisation producing the MatMulNBits layout (used by exporters and tests)."""
    n, k = w.shape
    if k % block:  # MatMulNBits pads the last K block with zeros
        w = torch.cat([w.float(), torch.zeros(n, block - k % block)], 1)
        k = w.shape[1]
    wb = w.float().view(n, k // block, block)
    if symmetric:
        amax = wb.abs().amax(-1).clamp_min(1e-8)
        scales = amax / 7.0
        codes = torch.clamp(torch.round(wb / scales[:, :, None]) + 8, 0, 15).to(torch.uint8)
        zp = None
    else:
        mn, mx = wb.amin(-1), wb.amax(-1)
        scales = ((mx - mn) / 15.0).clamp_min(1e-8)
        zpv = torch.clamp(torch.round(-mn / scales), 0, 15)
        codes = torch.clamp(torch.round(wb / scales[:, :, None]) + zpv[:, :, None], 0, 15).to(torch.uint8)
        kb = k // block
        zpi = zpv.to(torch.uint8)
        if kb % 2:
            zpi = torch.cat([zpi, torch.zeros(n, 1, dtype=torch.uint8)], dim=1)
        zp = (zpi[:, 0::2] | (zpi[:, 1::2] << 4)).contiguous()
    q = (codes[:, :, 0::2] | (codes[:, :, 1::2] << 4)).contiguous()
    return q, scales, zp


def moe_route(router_logits, k, renormalize=True, groups=1, keep=1, bias=None, score="softmax", group_best=1):
    """``groups`` > 1: only experts of the ``keep`` groups of neighbours whose ``group_best`` best experts score highest together can be
    chosen.  ``score`` "softmax": of logits plus ``bias``; "sigmoid": of the logits, and ``bias`` corrects the scores that are compared
    but not the weights."""
    logits = router_logits.float()
    if score == "sigmoid":
        probs = torch.sigmoid(logits)
        ranked = probs if bias is None else probs + bias
    else:
        ranked = probs = torch.softmax(logits if bias is None else logits + bias, dim=-1)
    if groups > 1:
        best = ranked.view(probs.shape[0], groups, -1)
        best = torch.topk(best, min(group_best, best.shape[-1]), dim=-1).values.sum(-1)
        kept = torch.zeros_like(best, dtype=torch.bool).scatter_(1, torch.topk(best, keep, dim=-1).indices, True)
        ranked = ranked.masked_fill(~kept.repeat_interleave(probs.shape[1] // groups, 1), float("-inf"))
    ids = torch.topk(ranked, k, dim=-1).indices
    w = probs.gather(1, ids)
    if renormalize:
        w = w / (w.sum(-1, keepdim=True) + (1e-20 if score == "sigmoid" else 0.0))
    return ids.to(torch.int32), w


# ------------------------------------------------------------------------------------------
# models with a mixer per layer (ops/hybrid.py)
# ------------------------------------------------------------------------------------------
def gelu_tanh(z):
    return torch.nn.functional.gelu(z, approximate="tanh")


def gated_act(act, g, u):
    """``act``: ops.hybrid.Act of a gate and an up value."""
    if act.kind == "clamp_glu":
        g, u = g.clamp(max=act.a), u.clamp(-act.a, act.a)
        return g * torch.sigmoid(1.702 * g) * (u + 1)
    return {"silu": torch.nn.functional.silu, "gelu_tanh": gelu_tanh}[act.kind](g) * u


def plain_act(v, act):
    """``act``: ops.hybrid.Act of one value."""
    if act.kind == "relu2":
        return torch.relu(v).pow(2)
    if act.kind == "xielu":
        return v / 2 + torch.where(v > 0, act.a * v * v, act.b * (torch.expm1(v.clamp(max=0)) - v))
    return v


def act_mul_packed(gate_up, half, act, out_dtype=None):
    """Gated activation over columns interleaved by :func:`pack_gate_up`."""
    t, n = gate_up.shape
    y = gate_up.float().view(t, n // (2 * half), 2, half)
    return gated_act(act, y[:, :, 0], y[:, :, 1]).reshape(t, n // 2).to(out_dtype or gate_up.dtype)


def hyper_step(x, y=None, mix=None, out_w=None, in_w=None, norm=None):
    """Streams x [T, S, W] fp32 -> (streams after folding y in, normed read-out u [T, W] fp32)."""
    if y is not None:
        x = torch.einsum("tsw,sq->tqw", x, mix) + out_w[None, :, None] * y.float()[:, None, : x.shape[2]]
    u = x.sum(1) if in_w is None else torch.einsum("tsw,s->tw", x, in_w)
    if norm is not None:
        u = torch.tanh(norm.alpha * u) * norm.w + norm.b
    return x, u


def step_entries(si):
    """(entry, first row, rows, position of the first row, state slot) of every sequence of a step plan."""
    nd = si.num_decode
    cu = si.cu_q[: si.num_prefill_seqs + 1].tolist()
    ctx, slots = si.ctx_len[: nd + si.num_prefill_seqs].tolist(), si.state_slot[: nd + si.num_prefill_seqs].tolist()
    for e, (c, slot) in enumerate(zip(ctx, slots)):
        base, n = (e, 1) if e < nd else (nd + cu[e - nd], cu[e - nd + 1] - cu[e - nd])
        if n > 0 and c > 0:
            yield e, base, n, c - n, slot


def token_shift(u, amount, prev, si):
    """u [T, W] fp32 -> shifted copy; prev [slots, W] holds every sequence's last row and is advanced."""
    out = u.clone()
    for _, base, n, start, slot in step_entries(si):
        rows = u[base:base + n]
        first = prev[slot] if start > 0 else torch.zeros_like(rows[0])
        before = torch.cat([first[None], rows[:-1]])
        out[base:base + n] = rows + (before - rows) * amount
        prev[slot] = rows[-1]
    return out


def hgrn2(qfv, bias, low, state, out, heads, dim, vdim, si):
    """Raw head outputs of the step's rows into out [T, heads * vdim]; state [slots, heads, vdim, rows >= dim] is advanced."""
    t = qfv.shape[0]
    hd = heads * dim
    q = torch.nn.functional.silu(qfv[:, :hd]).view(t, heads, dim)
    f = (low + (1 - low) * torch.sigmoid(qfv[:, hd:2 * hd] + bias)).view(t, heads, dim)
    v = qfv[:, 2 * hd:2 * hd + heads * vdim].view(t, heads, vdim)
    for _, base, n, start, slot in step_entries(si):
        s = state[slot, :, :, :dim].clone() if start > 0 else torch.zeros(heads, vdim, dim)
        for r in range(base, base + n):
            s = s * f[r][:, None, :] + v[r][:, :, None] * (1 - f[r])[:, None, :]
            out[r, : heads * vdim] = torch.einsum("hvd,hd->hv", s, q[r]).reshape(-1)
        state[slot, :, :, :dim] = s


def rms(x, w, eps, groups=1):
    """``groups``: equal consecutive parts with a root mean square each."""
    if groups > 1:
        parts = x.unflatten(-1, (groups, -1))
        return (parts * torch.rsqrt(parts.pow(2).mean(-1, keepdim=True) + eps)).flatten(-2) * w
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


def head_rmsnorm(x, w, eps, heads, n, out_dtype=None, gate=None, gate_act="silu"):
    """w: None, [n] for every head, or [heads * n]."""
    y = x[:, : heads * n].float().view(-1, heads, n)
    y = rms(y, 1.0 if w is None else w if w.numel() == n else w.view(heads, n), eps).reshape(x.shape[0], heads * n)
    if gate is not None:
        y = y * (torch.sigmoid(gate.float()) if gate_act == "sigmoid" else torch.nn.functional.silu(gate.float()))
    return y.to(out_dtype or x.dtype)


def norm_step(x, y, post):
    """x + post(y) for rows of y, or the weighted sum of a token's expert rows (ops.hybrid.ExpertRows); y as it is without post.
    ops.hybrid.GatedRows: those times the sigmoid of a gate, coordinate by coordinate."""
    if y is None:
        return x
    if hasattr(y, "gate_bias"):
        w = x.shape[1]
        inner = norm_step(torch.zeros_like(x), y.rows, None)
        if y.bias is not None:
            inner = inner + y.bias
        return x + inner * torch.sigmoid(y.gate[:, :w].float() + y.gate_bias)
    if not torch.is_tensor(y):
        rows = (y.rows[y.pos.long()].float() * y.weight[:, :, None]).sum(1)
        if y.shared is not None:
            w = min(rows.shape[1], y.shared.shape[1])
            rows = rows[:, :w] + torch.sigmoid(y.gate)[:, None] * y.shared[:, :w].float()
        y = rows
    y = y[:, : x.shape[1]].float()
    return x + (rms(y, post.w, post.eps, post.groups) if post is not None else y)


def short_conv(u, w, state, si):
    """u [T, C] fp32 -> sum_j w[j] u_(t - taps + 1 + j) along every sequence; state [slots, taps - 1, C] is advanced."""
    taps, out = w.shape[0], torch.empty_like(u)
    for _, base, n, start, slot in step_entries(si):
        before = state[slot].clone()
        before[: max(0, taps - 1 - start)] = 0
        rows = torch.cat([before, u[base:base + n]])
        out[base:base + n] = sum(w[j] * rows[j:j + n] for j in range(taps))
        if taps > 1:
            state[slot] = rows[-(taps - 1):]
    return out


def rotate_half(x, pos, freq):
    """x [T, heads, d]: dimension i turns with i + len(freq) by pos * freq[i]; dimensions past 2 len(freq) pass."""
    half = freq.numel()
    a = pos.double()[:, None] * freq[None, :]
    c, s = torch.cos(a).float()[:, None], torch.sin(a).float()[:, None]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


def conv_rope_append(u, w, bias, state, q, pool, freq, si, nq, nk, nv, d, dv, dp, vp):
    t, n = si.num_tokens, (nq + nk) * d + nv * dv
    y = short_conv(u[:, :n].float() + bias, w, state, si)
    x = rotate_half(y[:, :(nq + nk) * d].view(t, nq + nk, d), si.positions[:t], freq)
    q.view(t, nq, dp)[..., :d] = x[:, :nq].to(q.dtype)
    live = si.slots[:t] >= 0
    page, off = (si.slots[:t][live] // PAGE).long(), (si.slots[:t][live] % PAGE).long()
    keys, values = diff_pages(pool, nk, nv, dp, vp)
    keys[page, :, off, :d] = x[live, nq:].to(pool.dtype)
    values[page, :, off, :dv] = y[live, (nq + nk) * d:].view(-1, nv, dv).to(pool.dtype)


def diff_pages(pool, nk, nv, dp, vp):
    """Views of a pool of pages [nk][16][dp] | [nv][16][vp]: keys [pages, nk, 16, dp], values [pages, nv, 16, vp]."""
    k = nk * PAGE * dp
    return pool[:, :k].view(-1, nk, PAGE, dp), pool[:, k:k + nv * PAGE * vp].view(-1, nv, PAGE, vp)


def conv_unit_gates(u, w, state, ab, a_log, dt_bias, qk, v, gates, si, nk, nv, d, dv):
    t = si.num_tokens
    y = torch.nn.functional.silu(short_conv(u[:, :2 * nk * d + nv * dv].float(), w, state, si))
    x = y[:, :2 * nk * d].view(t, 2, nk, d)
    x = x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)
    x[:, 0] *= d ** -0.5
    qk[:t] = x.reshape(t, -1)
    v[:t] = y[:, 2 * nk * d:].to(v.dtype)
    gates[:t, :, 0] = -torch.exp(a_log) * torch.nn.functional.softplus(ab[:, :nv] + dt_bias)
    gates[:t, :, 1] = torch.sigmoid(ab[:, nv:2 * nv])


def delta_rule(qk, v, gates, state, out, heads, groups, dim, vdim, si):
    t, per = qk.shape[0], heads // groups
    q, k = (x.repeat_interleave(per, 1) for x in qk.view(t, 2, groups, dim).unbind(1))
    vv = v.float().view(t, heads, vdim)
    for _, base, n, start, slot in step_entries(si):
        s = state[slot, :, :, :dim].clone() if start > 0 else torch.zeros(heads, vdim, dim)
        for r in range(base, base + n):
            s = s * torch.exp(gates[r, :, 0])[:, None, None]
            w = gates[r, :, 1][:, None] * (vv[r] - torch.einsum("hvd,hd->hv", s, k[r]))
            s = s + w[:, :, None] * k[r][:, None, :]
            out[r, : heads * vdim] = torch.einsum("hvd,hd->hv", s, q[r]).reshape(-1)
        state[slot, :, :, :dim] = s


def diff_attention(q, out, pool, si, hq, hkv, d, dv, dp, vp, scale, lam, eps, gain, window, keep):
    keys, values = diff_pages(pool, 2 * hkv, hkv, dp, vp)
    for e, base, n, start, _ in step_entries(si):
        ctx = start + n
        lo = max(0, start - window + 1) if window > 0 else 0
        i, j = torch.arange(start, ctx)[:, None], torch.arange(ctx)[None, :]
        seen = j <= i
        if window > 0:
            seen &= (i - j < window) | (j < keep)
        near = (torch.arange(ctx) >= lo) | (torch.arange(ctx) < keep)      # pages in between may be gone
        j = j[0][near]
        page, off = si.page_table[e].long()[j // PAGE], j % PAGE
        k = keys[page, :, off, :d].float().view(-1, hkv, 2, d).repeat_interleave(hq // hkv, 1)
        v = values[page, :, off, :dv].float().repeat_interleave(hq // hkv, 1)
        s = torch.einsum("nhmd,khmd->hmnk", q[base:base + n].view(n, hq, 2, dp)[..., :d].float(), k) * scale
        p = torch.softmax(s.masked_fill(~seen[:, near], float("-inf")), -1)
        a = torch.einsum("hmnk,khd->mnhd", p, v)
        out[base:base + n].view(n, hq, vp)[..., :dv] = rms(a[0] - lam * a[1], gain, eps).to(out.dtype)


def rotate_pairs(x, pos, freq):
    """x [T, heads, 2 len(freq)]: dimension 2i turns with 2i + 1 by pos * freq[i]."""
    a = pos.double()[:, None] * freq[None, :]
    c, s = torch.cos(a).float()[:, None], torch.sin(a).float()[:, None]
    u, v = x[..., 0::2].float(), x[..., 1::2].float()
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)


def latent_append(row, latent, w, eps, slots, pool, rank, rope=None):
    """RMS norm of columns latent .. latent + rank, written to the rows' slots of pool [pages, 16, ld]; ``rope``: ops.hybrid.LatentRope."""
    y = row[:, latent:latent + rank].float()
    y = (y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + eps) * w).to(pool.dtype)
    flat = pool.view(-1, pool.shape[-1])
    live = slots >= 0
    at = slots[live].long()
    flat[at, :rank] = y[live]
    if rope is None:
        return
    t, rot = row.shape[0], 2 * rope.freq.numel()
    up8 = lambda n: n + (-n) % 8
    pos, part = rope.positions[:t], latent + up8(rank)
    flat[at, up8(rank):up8(rank) + rot] = rotate_pairs(row[:, None, part:part + rot], pos, rope.freq)[live, 0].to(pool.dtype)
    dp, step = up8(rope.dim), up8(rope.dim) + up8(rot)
    q = row[:, : rope.heads * step].unflatten(1, (rope.heads, step))[..., dp:dp + rot]
    turned = rotate_pairs(q, pos, rope.freq).to(row.dtype)
    if rope.split > 0:
        rope.q_out[: rope.split * rope.heads, rope.q_col:rope.q_col + rot] = turned[: rope.split].reshape(-1, rot)
    q[rope.split:] = turned[rope.split:]


def latent_attention(q, out, pool, si, heads, rank, scale, window, vrank=None, gate=None):
    """q [T * heads, >= rank]: every head attends to the page rows of its sequence (keys, and values in the first vrank columns)."""
    vrank = rank if vrank is None else vrank
    for e, base, n, start, _ in step_entries(si):
        ctx = start + n
        lo = max(0, start - window + 1) if window > 0 else 0
        pages = si.page_table[e, lo // PAGE:(ctx + PAGE - 1) // PAGE].long()
        c = pool[pages].reshape(-1, pool.shape[-1])[: ctx - lo // PAGE * PAGE, :rank].float()
        j = torch.arange(lo // PAGE * PAGE, ctx)
        i = torch.arange(start, ctx)
        seen = j[None, :] <= i[:, None]
        if window > 0:
            seen &= i[:, None] - j[None, :] < window
        qs = q[base * heads:(base + n) * heads, :rank].float().view(n, heads, rank)
        s = torch.einsum("nhr,kr->nhk", qs, c) * scale
        p = torch.softmax(s.masked_fill(~seen[:, None, :], float("-inf")), -1)
        o = torch.einsum("nhk,kr->nhr", p, c[:, :vrank])
        if gate is not None:
            o = o * torch.sigmoid(gate[base:base + n].float())[..., None]
        out[base * heads:(base + n) * heads, :vrank] = o.reshape(n * heads, vrank).to(out.dtype)


# ------------------------------------------------------------------------------------------
# attention whose values are its keys, and recurrences with one decay per head (ops/hybrid.py)
# ------------------------------------------------------------------------------------------
def tied_pages(pool, hkv, dp):
    """Views of a pool of pages [hkv][16][dp] | [16] factors: keys [pages, hkv, 16, dp], factors [pages, 16] fp32."""
    n = hkv * PAGE * dp
    tail = PAGE * 4 // pool.element_size()
    return pool[:, :n].view(-1, hkv, PAGE, dp), pool.view(torch.float32)[:, n * pool.element_size() // 4:(n + tail) * pool.element_size() // 4]


def tied_append(row, q_bias, k_bias, q_gain, eps, factor, q, pool, slots, hq, hkv, d, dp):
    t = row.shape[0]
    qs, ks = row[:, : hq * d].float(), row[:, hq * d:(hq + hkv) * d].float()
    qs, ks = qs if q_bias is None else qs + q_bias, ks if k_bias is None else ks + k_bias
    pad = lambda x: torch.nn.functional.pad(x, (0, dp - d))
    q[:t] = pad(rms(qs, q_gain, eps).view(t, hq, d)).to(q.dtype).reshape(t, -1)
    live = slots[:t] >= 0
    page, off = (slots[:t][live] // PAGE).long(), (slots[:t][live] % PAGE).long()
    keys, factors = tied_pages(pool, hkv, dp)
    keys[page, :, off] = pad(ks.view(t, hkv, d))[live].to(pool.dtype)
    factors[page, off] = (torch.rsqrt(ks.pow(2).mean(-1) + eps) * factor)[live]


def tied_attention(q, out, pool, si, hq, hkv, d, dp, cap, slope, sink, window, gate):
    keys, factors = tied_pages(pool, hkv, dp)
    for e, base, n, start, _ in step_entries(si):
        ctx = start + n
        lo = max(0, start - window + 1) if window > 0 else 0
        j = torch.arange(lo, ctx)
        dist = torch.arange(start, ctx)[:, None] - j[None, :]
        seen = dist >= 0
        if window > 0:
            seen &= dist < window
        page, off = si.page_table[e].long()[j // PAGE], j % PAGE
        k = keys[page, :, off, :d].float().repeat_interleave(hq // hkv, 1)
        s = torch.einsum("nhd,khd->hnk", q[base:base + n].view(n, hq, dp)[..., :d].float(), k) * factors[page, off]
        if cap > 0:
            s = cap * torch.tanh(s)
        if slope is not None:
            s = s - slope[:, None, None] * dist
        s = s.masked_fill(~seen, float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink[:, None, None].expand(-1, n, 1)], -1)
        p = torch.softmax(s, -1)[..., : j.numel()]
        o = torch.einsum("hnk,khd->nhd", p, k)
        if gate is not None:
            o = o * torch.sigmoid(gate[base:base + n, :hq].float())[..., None]
        out[base:base + n] = torch.nn.functional.pad(o, (0, dp - d)).to(out.dtype).reshape(n, -1)


def turn_table(positions, freq, out):
    """out [T, len(freq), 2] fp32: cosine and sine of position x freq."""
    a = positions.double()[:, None] * freq[None, :]
    out[: a.shape[0], :, 0], out[: a.shape[0], :, 1] = torch.cos(a).float(), torch.sin(a).float()


def memory_gates(logits, bias, cap, heads):
    """(log input gate, log forget gate) [T, heads] of logits [T, >= 2 heads] (input | forget)."""
    z = cap * torch.tanh((logits[:, : 2 * heads].float() + bias) / cap)
    return z[:, :heads], torch.nn.functional.logsigmoid(z[:, heads:])


def decay_memory(row, turns, logits, bias, cap, decay, state, peak, out, heads, dim, vdim, q_scale, k_scale, si):
    t, hd = row.shape[0], heads * dim
    q, k = row[:, :hd].float().view(t, heads, dim), row[:, hd:2 * hd].float().view(t, heads, dim)
    v = row[:, 2 * hd:2 * hd + heads * vdim].float().view(t, heads, vdim)
    if turns is not None:
        half = turns.shape[1]
        c, s = turns[:t, None, :, 0], turns[:t, None, :, 1]
        turn = lambda x: torch.cat([x[..., :half] * c - x[..., half:2 * half] * s, x[..., half:2 * half] * c + x[..., :half] * s, x[..., 2 * half:]], -1)
        q, k = turn(q), turn(k)
    q, k = q * q_scale, k * k_scale
    gated = logits is not None
    if gated:
        gi, gf = memory_gates(logits, bias, cap, heads)
        v = torch.cat([v, torch.ones(t, heads, 1)], -1)              # one more value column holds the normalizer
    for _, base, n, start, slot in step_entries(si):
        s = state[slot, :, :, :dim].clone() if start > 0 else torch.zeros(heads, v.shape[2], dim)
        m = peak[slot].clone() if gated and start > 0 else torch.zeros(heads)
        for r in range(base, base + n):
            if gated:
                new = torch.maximum(gf[r] + m, gi[r])
                keep, take, m = torch.exp(gf[r] + m - new), torch.exp(gi[r] - new), new
            else:
                keep, take = decay[0], torch.ones(heads)
            s = s * keep[:, None, None] + (take[:, None] * v[r])[:, :, None] * k[r][:, None, :]
            o = torch.einsum("hvd,hd->hv", s, q[r])
            if gated:
                o = o[:, :vdim] / (torch.maximum(o[:, vdim].abs(), torch.exp(-m)) + 1e-6)[:, None]
            out[r, : heads * vdim] = o.reshape(-1)
        state[slot, :, :, :dim] = s
        if gated:
            peak[slot] = m
