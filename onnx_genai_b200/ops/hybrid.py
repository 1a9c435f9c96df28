"""Ops of models that choose a mixer per layer (csrc/kernels/hybrid.cu, recurrent.cu, latent_attention.cu, short_conv.cu,
delta_rule.cu, diff_attention.cu, decay_memory.cu, tied_attention.cu): hyper-connected residual streams with a Dynamic-Tanh norm and
token shift, one residual stream with RMS norms before (and behind) a sublayer, convolutions of what a sublayer reads and gates of
what it adds, HGRN2, gated delta-rule and one-decay-per-head recurrences over per-sequence state, short causal convolutions, attention
over paged latents with or without a rotated part, over paged keys that are the values too, differential attention over paged keys
and values, products with activations, batched per-head products, and the fp32 matrix product of the 32-bit engine.

CUDA tensors run the kernels; CPU tensors run the statements in :mod:`onnx_genai_b200.ops.reference`, as the other ops do.
``si`` is the step's :class:`~onnx_genai_b200.models.decoder.StepInputs`.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from . import _native, _ptr, _stream, _timed, backed_pages, launch_counts, reference, status_word
from . import PAGE, gemm

P, I, F, L = _native.P, _native.I, _native.F, _native.L
_native.register("ogb_hyper_step", [P] * 13 + [I] * 6 + [P] * 5 + [I] * 4 + [P, P])
_native.register("ogb_embed_streams", [P, P, P, I, I, I, I, P, F, F, P, I, I, P, P])
_native.register("ogb_latent_append", [P, I, I, P, F, P, P, I, I, I, L, P, P, P] + [I] * 7 + [P, P])
_native.register("ogb_latent_attention", [P] * 9 + [I] * 10 + [L, I, F, I, P, P, P, I, P, P])
_native.register("ogb_paged_prefill_chunks_bf16", [P] * 9 + [I] * 4 + [L] + [I] * 9 + [F, I, P, P])
_native.register("ogb_gemm_bf16_act", [P] * 3 + [I] * 7 + [F, F, I, P, P])
_native.register("ogb_gemm_f32_act", [P] * 3 + [I] * 7 + [F, F, P])
_native.register("ogb_latent_gather", [P, P, P, P, I, I, L, I, I, I, P, P, P, P])
_native.register("ogb_latent_set_tc", [I])
_native.register("ogb_gemm_bf16_paged", [P, P, P, I, I, I, I, I, I, P, P])
_native.register("ogb_hgrn2_state_rows", [I])
_native.register("ogb_hgrn2", [P] * 5 + [I] * 5 + [P] * 3 + [I] * 5 + [P, P, I, P, P])
_native.register("ogb_head_rmsnorm", [P, P, I, F, P, I, I, I, I, I, P, I, I, I, P])
_native.register("ogb_norm_step", [P] * 13 + [F] + [I] * 10 + [L, I, P, P])
_native.register("ogb_norm_conv_step", [P] * 17 + [F] + [I] * 12 + [L] + [P] * 5 + [I] * 4 + [P, P])
_native.register("ogb_turn_table", [P, P, P, I, I, P])
_native.register("ogb_tied_append", [P, I, P, P, P, F, F, P, I, P, P, L, L] + [I] * 6 + [P, P])
_native.register("ogb_tied_attention", [P] * 11 + [I] * 3 + [L, L] + [I] * 8 + [F, I, P, P, P, I, P, P])
_native.register("ogb_tied_set_tc", [I])
_native.register("ogb_decay_memory", [P, I, P, I, P, I, P, F] + [P] * 4 + [I] * 4 + [F, F] + [P] * 5 + [I] * 4 + [P, I, P, P])
_native.register("ogb_decay_block_floats", [I] * 4)
_native.register("ogb_conv_rope_append", [P, I, P, P, P, I, P, I, P, P, P, L, L] + [I] * 8 + [P] * 5 + [I] * 4 + [P, P])
_native.register("ogb_conv_unit_gates", [P, I, P, P, I, P, I] + [P] * 5 + [I] * 4 + [P] * 5 + [I] * 4 + [P, P])
_native.register("ogb_delta_rule", [P] * 5 + [I] * 4 + [P] * 5 + [I] * 4 + [P, I, P, P])
_native.register("ogb_delta_block_floats", [I] * 4)
_native.register("ogb_diff_attention", [P] * 8 + [I] * 3 + [L, L] + [I] * 10 + [F] * 4 + [I, P, P, P, I, P, P])
_native.register("ogb_diff_set_tc", [I])
_native.register("ogb_act_mul_packed", [P, P, I, I, I, I, F, F, I, P])

ACTS = {"none": 0, "silu": 1, "gelu_tanh": 2, "relu2": 3, "clamp_glu": 4, "xielu": 5}
_ELEM = {torch.float32: 0, torch.bfloat16: 1}


@dataclass
class DynamicTanh:
    """tanh(alpha x) w + b, all fp32 (alpha is a one-element tensor)."""
    alpha: torch.Tensor
    w: torch.Tensor
    b: torch.Tensor


@dataclass
class HyperConnection:
    """Weights of one sublayer over S residual streams, fp32: reads sum_s read[s] x_s, writes
    x_t <- sum_s mix[s, t] x_s + write[t] y."""
    read: torch.Tensor
    write: torch.Tensor
    mix: torch.Tensor


@dataclass
class RmsNorm:
    """x / sqrt(mean(x^2) + eps) w; w fp32.  ``groups``: equal consecutive parts of x, each over its own root mean square."""
    w: torch.Tensor
    eps: float
    groups: int = 1


@dataclass
class ExpertRows:
    """A sublayer's output that is still spread over expert rows: token t's is sum_j weight[t, j] rows[pos[t, j]], and a shared
    expert's row times sigmoid(gate[t]) (a column of fp32 logits) where there is one."""
    rows: torch.Tensor
    pos: torch.Tensor
    weight: torch.Tensor
    shared: torch.Tensor | None = None
    gate: torch.Tensor | None = None


@dataclass
class GatedRows:
    """A sublayer's output (``rows``: a row per token, or :class:`ExpertRows`; plus ``bias`` [W] fp32 where given) that reaches the residual
    times sigmoid(gate + gate_bias), coordinate by coordinate: gate [T, ld], gate_bias [W] fp32."""
    rows: object
    gate: torch.Tensor
    gate_bias: torch.Tensor
    bias: torch.Tensor | None = None


@dataclass(frozen=True)
class Act:
    """Activation of a feed-forward and its numbers.  Gated: silu, gelu_tanh, clamp_glu (a: limit); of one value: relu2, xielu
    (a, b: weights of its rising and its falling side)."""
    kind: str
    a: float = 0.0
    b: float = 0.0

    @property
    def gated(self) -> bool:
        return self.kind in ("silu", "gelu_tanh", "clamp_glu")

    @property
    def args(self):
        return ACTS[self.kind], float(self.a), float(self.b)


def as_act(act) -> Act:
    return act if isinstance(act, Act) else Act(act)


def state_rows(dim: int) -> int:
    """Row width at which the recurrence keeps a state of ``dim`` key channels."""
    for n in (64, 128, 256):
        if dim <= n:
            return n
    raise ValueError(f"recurrent key width {dim} is not supported (at most 256)")


@_timed("linear")
def linear(a, w, out, f32_out=False):
    """out = a @ w^T: bf16 on the tensor cores (fp32 results with ``f32_out``), fp32 operands in true fp32."""
    if not a.is_cuda:
        out.copy_(reference.gemm(a, w, out_dtype=out.dtype))
        return out
    if a.dtype == torch.bfloat16:
        return gemm(a, w, out=out, out_f32=f32_out)
    return linear_batched(a, w, out, 1, 0, 0)


@_timed("linear_batched")
def linear_batched(a, w, out, batch, a_step, c_step):
    """out[:, z*c_step : +N] = a[:, z*a_step : +K] @ w[z*N : +N]^T for every z < batch; w is [batch * N, K]."""
    m, k = a.shape[0], w.shape[1]
    n = w.shape[0] // batch
    if not a.is_cuda:
        for z in range(batch):
            out[:, z * c_step:z * c_step + n] = reference.gemm(a[:, z * a_step:z * a_step + k], w[z * n:(z + 1) * n], out_dtype=out.dtype)
        return out
    lib = _native.load()
    if a.dtype == torch.bfloat16:
        rc = lib.ogb_gemm_bf16_batched(a.data_ptr(), w.data_ptr(), out.data_ptr(), m, n, k, a.stride(0), w.stride(0), out.stride(0), batch,
                                       a_step, c_step, status_word().data_ptr(), _stream())
        _native.check(rc, "ogb_gemm_bf16_batched")
        launch_counts["gemm_bf16_tcgen05"] += 1
    else:
        rc = lib.ogb_gemm_f32(a.data_ptr(), w.data_ptr(), out.data_ptr(), m, n, k, a.stride(0), w.stride(0), out.stride(0), batch, a_step,
                              c_step, _stream())
        _native.check(rc, "ogb_gemm_f32")
        launch_counts["gemm_f32"] += 1
    return out


@_timed("gated_linear")
def gated_linear(a, w_packed, half, act, out, scratch=None):
    """out = act(a @ gate^T, a @ up^T) over a weight packed by ``ops.pack_gate_up``; ``act``: a gated :class:`Act` or its name.  bf16 in
    one product with the gate in its epilogue, fp32 through ``scratch`` [rows, 2 * inter]."""
    act = as_act(act)
    if not a.is_cuda:
        out.copy_(reference.act_mul_packed(reference.gemm(a, w_packed, out_dtype=torch.float32), half, act, out.dtype))
        return out
    m, n = a.shape[0], w_packed.shape[0]
    if a.dtype == torch.bfloat16:
        rc = _native.load().ogb_gemm_bf16_act(a.data_ptr(), w_packed.data_ptr(), out.data_ptr(), m, n, a.shape[1], a.stride(0), w_packed.stride(0),
                                              out.stride(0), *act.args, 2 * half, status_word().data_ptr(), _stream())
        _native.check(rc, "ogb_gemm_bf16_act")
        launch_counts["gemm_bf16_tcgen05"] += 1
        return out
    gu = scratch[:m, :n]
    assert gu.is_contiguous() and out.is_contiguous()
    linear(a, w_packed, gu)
    return act_mul_packed(gu, half, act, out)


def act_mul_packed(gate_up, half, act, out):
    """Gated activation over columns packed by ``ops.pack_gate_up`` (contiguous rows)."""
    m, n = gate_up.shape
    rc = _native.load().ogb_act_mul_packed(gate_up.data_ptr(), out.data_ptr(), m, n // 2, half, *as_act(act).args, _ELEM[out.dtype], _stream())
    _native.check(rc, "ogb_act_mul_packed")
    launch_counts["act_mul_packed"] += 1
    return out


@_timed("act_linear")
def act_linear(a, w, act, out):
    """out = act(a @ w^T) for an :class:`Act` of one value."""
    act = as_act(act)
    if not a.is_cuda:
        out.copy_(reference.plain_act(reference.gemm(a, w, out_dtype=torch.float32), act).to(out.dtype))
        return out
    m, n, k = a.shape[0], w.shape[0], w.shape[1]
    lib, ld = _native.load(), (a.stride(0), w.stride(0), out.stride(0))
    if a.dtype == torch.bfloat16:
        rc = lib.ogb_gemm_bf16_act(a.data_ptr(), w.data_ptr(), out.data_ptr(), m, n, k, *ld, *act.args, 0, status_word().data_ptr(), _stream())
        _native.check(rc, "ogb_gemm_bf16_act")
        launch_counts["gemm_bf16_tcgen05"] += 1
    else:
        rc = lib.ogb_gemm_f32_act(a.data_ptr(), w.data_ptr(), out.data_ptr(), m, n, k, *ld, *act.args, _stream())
        _native.check(rc, "ogb_gemm_f32_act")
        launch_counts["gemm_f32"] += 1
    return out


@_timed("embed_streams")
def embed_streams(ids, table, x, norm: RmsNorm | None = None, copy=None, scale=1.0):
    """Every stream of row t of x [T, S, W] (fp32) becomes the embedding of ids[t] times ``scale``, normed where ``norm`` is given; so does
    row t of ``copy`` [T, W]."""
    t, s, w = x.shape
    if not x.is_cuda:
        rows = table[ids[:t].long()].float() * scale
        if norm is not None:
            rows = reference.rms(rows, norm.w, norm.eps)
        x.copy_(rows[:, None, :].expand(-1, s, -1))
        if copy is not None:
            copy.copy_(rows)
        return x
    rc = _native.load().ogb_embed_streams(ids.data_ptr(), table.data_ptr(), x.data_ptr(), t, s, w, table.shape[0], _ptr(norm.w if norm is not None else None),
                                          float(norm.eps) if norm is not None else 0.0, float(scale), _ptr(copy), copy.stride(0) if copy is not None else 0,
                                          _ELEM[table.dtype], status_word().data_ptr(), _stream())
    _native.check(rc, "ogb_embed_streams")
    launch_counts["embed_streams"] += 1
    return x


@_timed("hyper_step")
def hyper_step(x_in, x_out, y, written: HyperConnection | None, read, norm: DynamicTanh | None, h, si, shift=None, prev=None, gather=None):
    """Fold the last sublayer's output ``y`` into the streams (weights ``written``; x_in -> x_out), read the next sublayer's
    input (weights ``read``, None: the sum), norm it and shift it by a token where ``shift`` is given (state ``prev`` [slots, W]).
    ``gather``: h gets the rows it names only, and nothing is written back."""
    rows = h.shape[0] if h is not None else x_in.shape[0]
    if not x_in.is_cuda:
        src = x_in if gather is None else x_in[gather.long()]
        ys = y if (y is None or gather is None) else y[gather.long()]
        x, u = reference.hyper_step(src, ys, written.mix if y is not None else None, written.write if y is not None else None, read, norm)
        if y is not None and x_out is not None:
            x_out.copy_(x)
        if h is not None:
            if shift is not None:
                u = reference.token_shift(u, shift, prev, si)
            h[:, : u.shape[1]] = u.to(h.dtype)
        return h
    elem = _ELEM[h.dtype if h is not None else y.dtype]
    assert y is None or h is None or y.dtype == h.dtype
    total, s, w = x_in.shape
    rc = _native.load().ogb_hyper_step(
        x_in.data_ptr(), _ptr(x_out), _ptr(y), _ptr(written.mix if y is not None else None), _ptr(written.write if y is not None else None),
        _ptr(read), _ptr(norm.alpha if norm is not None else None), _ptr(norm.w if norm is not None else None),
        _ptr(norm.b if norm is not None else None), _ptr(shift), _ptr(prev), _ptr(h), _ptr(gather), rows, total, s, w,
        y.stride(0) if y is not None else 0, h.stride(0) if h is not None else 0, si.ctx_len.data_ptr(), _ptr(si.state_slot),
        si.cu_q.data_ptr(), si.tile_seq.data_ptr(), si.tile_q0.data_ptr(), si.num_decode, si.num_tiles,
        prev.shape[0] if prev is not None else 0, elem, status_word().data_ptr(), _stream())
    _native.check(rc, "ogb_hyper_step")
    launch_counts["hyper_step"] += 1
    return h


@_timed("latent_append")
def latent_append(row, latent, w, eps, slots, pool, rank, rope=None):
    """RMS-norm the latents in columns latent .. latent + rank of the projected rows [T, ld] and write them to their slots of pool
    [pages, 16, ld].  ``rope``: a :class:`LatentRope`, which turns the rows' rotated parts."""
    t = row.shape[0]
    if not row.is_cuda:
        reference.latent_append(row, latent, w, eps, slots[:t], pool, rank, rope)
        return
    assert pool.dtype == row.dtype
    turn = [0, 0, 0, 0, 0, 0, 0, 0, 0]
    if rope is not None:
        q = rope.q_out
        turn = [rope.freq.data_ptr(), rope.positions.data_ptr(), _ptr(q), rope.heads, rope.dim, 2 * rope.freq.numel(), q.stride(0) if q is not None else 0,
                rope.q_col, rope.split]
    rc = _native.load().ogb_latent_append(row.data_ptr(), row.stride(0), latent, w.data_ptr(), float(eps), slots.data_ptr(), pool.data_ptr(), t, rank,
                                          pool.shape[2], backed_pages(pool) * PAGE, *turn, _ELEM[row.dtype], status_word().data_ptr(), _stream())
    _native.check(rc, "ogb_latent_append")
    launch_counts["latent_append"] += 1


@dataclass
class LatentRope:
    """Rotated parts beside a latent.  A projected row holds ``heads`` queries of pad8(dim) + pad8(rot) columns, then the latent (in
    pad8(rank) columns) and the key part that all heads share; neighbours 2i, 2i + 1 of a part turn by position x freq[i].  Query parts
    go to columns q_col .. of q_out [T * heads, ld] for rows below ``split`` and stay where they are for the others."""
    freq: torch.Tensor           # fp64 [rot / 2]
    positions: torch.Tensor
    heads: int
    dim: int
    q_out: torch.Tensor | None
    q_col: int
    split: int


@_timed("latent_attention")
def latent_attention(q, out, pool, si, heads, rank, scale, window, splits=1, part_o=None, part_ml=None, counters=None, decode_only=False, vrank=None,
                     gate=None):
    """Rows (token, head) of q [T * heads, ld] over the latents of their sequences' pages; window <= 0: causal only.  The first ``rank``
    values of a page row are the key, the first ``vrank`` (None: all of them) the value.  ``gate`` [T, heads]: every head's output times
    the sigmoid.  ``counters``: zeroed int32 words, one per decode row and 16 heads, with which the last split of a row merges the
    splits.  ``decode_only``: leave the prefill rows to :func:`latent_prefill_expanded`."""
    vrank = rank if vrank is None else vrank
    if not q.is_cuda:
        reference.latent_attention(q, out, pool, si, heads, rank, scale, window, vrank, gate)
        return out
    lib, st = _native.load(), status_word().data_ptr()
    nd, npf, t = si.num_decode, si.num_prefill_seqs, si.num_tokens
    pages, mp = backed_pages(pool), si.page_table.shape[1]
    elem = _ELEM[q.dtype]
    sizes = (heads, rank, vrank, q.stride(0), out.stride(0), pool.shape[2], gate.stride(0) if gate is not None else 0, mp)
    if nd > 0:
        rc = lib.ogb_latent_attention(q.data_ptr(), out.data_ptr(), pool.data_ptr(), si.page_table.data_ptr(), si.ctx_len.data_ptr(), 0, 0, 0, _ptr(gate),
                                      nd, *sizes, 0, pages, int(window), float(scale), int(splits), _ptr(part_o), _ptr(part_ml), _ptr(counters), elem, st,
                                      _stream())
        _native.check(rc, "ogb_latent_attention")
        launch_counts["latent_decode"] += 1
    if npf > 0 and not decode_only:
        qp, op = q[nd * heads:], out[nd * heads:]
        rc = lib.ogb_latent_attention(qp.data_ptr(), op.data_ptr(), pool.data_ptr(), si.page_table[nd:].data_ptr(), si.ctx_len[nd:].data_ptr(),
                                      si.cu_q.data_ptr(), si.tile_seq.data_ptr(), si.tile_q0.data_ptr(), _ptr(gate[nd:] if gate is not None else None),
                                      t - nd, *sizes, si.num_tiles, pages, int(window), float(scale), 1, 0, 0, 0, elem, st, _stream())
        _native.check(rc, "ogb_latent_attention")
        launch_counts["latent_prefill"] += 1
    return out


def visible_pages(si, window):
    """KV pages that the prefill rows of a step can see, from the host's copy of the plan."""
    start = si.prefill_ctx - si.prefill_len
    lo = (start - window + 1).clip(0) // PAGE if window > 0 else 0
    return int(((si.prefill_ctx + PAGE - 1) // PAGE - lo).sum())


def latent_prefill_expanded(q, out, pool, kv_w, si, heads, kc, vc, q_head, dv, scale, window, pages, dense, kv, table, gate=None):
    """Prefill rows with keys and values expanded: the visible page rows are packed (``dense`` [16 * pages, ld]), one product with
    ``kv_w`` [heads * (kc key | vc value chunks) * 64, ld] writes pages of 64-column chunks (``kv`` [pages, heads, kc + vc, 16, 64]), and the
    paged prefill kernel of the dense decoders runs over them through ``table``.  q: heads of ``q_head`` columns, out: of ``dv``.  Worth it
    when many queries share a latent and the latent is wider than a head: a (query, key) pair then costs the head's widths in operations
    instead of the latent's."""
    nd, npf, t = si.num_decode, si.num_prefill_seqs, si.num_tokens
    lib, st = _native.load(), status_word().data_ptr()
    mp = si.page_table.shape[1]
    rc = lib.ogb_latent_gather(pool.data_ptr(), si.page_table[nd:].data_ptr(), si.ctx_len[nd:].data_ptr(), si.cu_q.data_ptr(), npf, mp,
                               backed_pages(pool), int(window), pool.shape[2], pages, dense.data_ptr(), table.data_ptr(), st, _stream())
    _native.check(rc, "ogb_latent_gather")
    rc = lib.ogb_gemm_bf16_paged(dense.data_ptr(), kv_w.data_ptr(), kv.data_ptr(), pages * PAGE, kv_w.shape[0], kv_w.shape[1], dense.stride(0),
                                 kv_w.stride(0), 64, st, _stream())
    _native.check(rc, "ogb_gemm_bf16_paged")
    rc = lib.ogb_paged_prefill_chunks_bf16(q[nd:].data_ptr(), out[nd:].data_ptr(), kv.data_ptr(), table.data_ptr(), si.ctx_len[nd:].data_ptr(),
                                           si.cu_q.data_ptr(), si.tile_seq.data_ptr(), si.tile_q0.data_ptr(), _ptr(gate[nd:] if gate is not None else None),
                                           si.num_tiles, npf, t - nd, mp, pages, heads, kc, vc, dv, q_head, dv, q.stride(0), out.stride(0),
                                           gate.stride(0) if gate is not None else 0, float(scale), int(window), st, _stream())
    _native.check(rc, "ogb_paged_prefill_chunks_bf16")
    launch_counts["latent_expand"] += 1
    launch_counts["paged_prefill_tc"] += 1


def segment_length(si, heads: int, vdim: int) -> int:
    """Tokens per segment of a step's prompts, 0 to run every chunk in one piece: chunks are cut while the (head, chunk) pairs
    leave much of the device empty (a segmented run goes over the gates twice)."""
    if si.num_prefill_seqs == 0 or si.prefill_len is None:
        return 0
    longest, per = int(si.prefill_len.max()), heads * max(1, -(-vdim // 128))
    if per * si.num_prefill_seqs >= 100 or longest < 256:
        return 0
    seg = 1 << (longest - 1).bit_length()
    while seg > 128 and per * int((-(-si.prefill_len // seg)).sum()) < 256:
        seg //= 2
    return seg if seg < longest else 0


@_timed("hgrn2")
def hgrn2(qfv, bias, low, state, out, heads, dim, vdim, si, segment=None, scratch=None, split=False):
    """Advance the recurrence over the step's rows: qfv [T, ld] fp32 (query, gate and value projections), state
    [slots, heads, vdim, state_rows(dim)] fp32 in place, raw head outputs to out [T, ld] fp32.  ``segment``: tokens per segment of
    the prompts (None: chosen, 0: whole); ``scratch(name, shape)`` provides fp32 scratch for segmented runs.
    ``split``: prompts in blocks on the tensor cores, fp32 factors split in two tf32 terms (v rounded to one)."""
    if not qfv.is_cuda:
        reference.hgrn2(qfv, bias, low, state, out, heads, dim, vdim, si)
        return out
    seg = segment_length(si, heads, vdim) if segment is None else segment
    nseg, us, ug = 0, None, None
    if seg > 0 and si.num_prefill_seqs > 0:
        nseg, rows = int((-(-si.prefill_len // seg)).sum()), state.shape[3]
        make = scratch or (lambda name, shape: torch.empty(*shape, dtype=torch.float32, device=qfv.device))
        us, ug = make("seg_state", (nseg, heads, vdim, rows)), make("seg_gate", (nseg, heads, rows))
    rc = _native.load().ogb_hgrn2(qfv.data_ptr(), bias.data_ptr(), low.data_ptr(), state.data_ptr(), out.data_ptr(), qfv.stride(0),
                                  out.stride(0), heads, dim, vdim, si.ctx_len.data_ptr(), si.state_slot.data_ptr(), si.cu_q.data_ptr(),
                                  si.num_decode, si.num_prefill_seqs, state.shape[0], seg if nseg else 0, nseg, _ptr(us), _ptr(ug),
                                  int(split), status_word().data_ptr(), _stream())
    _native.check(rc, "ogb_hgrn2")
    launch_counts["hgrn2"] += 1
    return out


@_timed("head_rmsnorm")
def head_rmsnorm(x, w, eps, out, heads, n, gate=None, gate_act="silu"):
    """RMS norm of each head's n columns of x [T, ld] (fp32) with a weight (None, [n] for every head, or [heads * n]), times silu or sigmoid
    (``gate_act``) of gate [T, heads * n] where given."""
    if not x.is_cuda:
        out[:, : heads * n] = reference.head_rmsnorm(x, w, eps, heads, n, out.dtype, gate, gate_act)
        return out
    step = n if w is not None and w.numel() != n else 0
    rc = _native.load().ogb_head_rmsnorm(x.data_ptr(), _ptr(w), step, float(eps), out.data_ptr(), x.shape[0], heads, n, x.stride(0), out.stride(0),
                                         _ptr(gate), gate.stride(0) if gate is not None else 0, int(gate_act == "sigmoid"), _ELEM[out.dtype], _stream())
    _native.check(rc, "ogb_head_rmsnorm")
    launch_counts["head_rmsnorm"] += 1
    return out


def _sublayer(y):
    """(output rows, kernel pointers, (k, ldy, lds, ldg, ldr), expert rows) of a sublayer's output: rows, :class:`ExpertRows`,
    :class:`GatedRows` of either, or None."""
    scaled, ldr = (0, 0, 0), 0
    if isinstance(y, GatedRows):
        scaled, ldr = (_ptr(y.bias), y.gate.data_ptr(), y.gate_bias.data_ptr()), y.gate.stride(0)
        assert y.gate.dtype == (y.rows.rows if isinstance(y.rows, ExpertRows) else y.rows).dtype
        y = y.rows
    if not isinstance(y, ExpertRows):
        return y, (_ptr(y), 0, 0, 0, 0, *scaled), (1, y.stride(0) if y is not None else 0, 0, 0, ldr), 0
    shared = (_ptr(y.shared), _ptr(y.gate))
    assert y.shared is None or (y.shared.dtype == y.rows.dtype and y.gate.dtype == torch.float32)
    lds, ldg = (y.shared.stride(0), y.gate.stride(0)) if y.shared is not None else (0, 0)
    return (y.rows, (y.rows.data_ptr(), y.pos.data_ptr(), y.weight.data_ptr(), *shared, *scaled), (y.pos.shape[1], y.rows.stride(0), lds, ldg, ldr),
            y.rows.shape[0])


@_timed("norm_step")
def norm_step(x, y, post: RmsNorm | None, norm: RmsNorm | None, h, gather=None):
    """x [T, W] fp32 += post(y) (None: y as it is); h = norm(x) (None: x).  ``y``: rows of the last sublayer's output, :class:`ExpertRows`,
    :class:`GatedRows`, or None.  ``gather``: h gets the rows it names only, and x stays as it is."""
    rows = h.shape[0] if h is not None else x.shape[0]
    if not x.is_cuda:
        new = reference.norm_step(x, y, post)
        if gather is None:
            x.copy_(new)
        else:
            new = new[gather.long()]
        if h is not None:
            h[:, : x.shape[1]] = (reference.rms(new, norm.w, norm.eps, norm.groups) if norm is not None else new).to(h.dtype)
        return h
    src, ptrs, (k, ldy, lds, ldg, ldr), y_rows = _sublayer(y)
    eps = norm.eps if norm is not None else post.eps if post is not None else 0.0
    assert post is None or (post.eps == eps and post.groups == 1)
    assert x.is_contiguous()
    rc = _native.load().ogb_norm_step(
        x.data_ptr(), *ptrs, _ptr(post.w if post is not None else None), _ptr(norm.w if norm is not None else None), _ptr(h), _ptr(gather), float(eps), rows,
        x.shape[0], x.shape[1], norm.groups if norm is not None else 1, k, ldy, lds, ldg, ldr, h.stride(0) if h is not None else 0, y_rows, _ELEM[h.dtype if h is not None else src.dtype],
        status_word().data_ptr(), _stream())
    _native.check(rc, "ogb_norm_step")
    launch_counts["norm_step"] += 1
    return h


@_timed("norm_conv_step")
def norm_conv_step(x_in, x_out, y, add, norm: RmsNorm, conv, state, h, si, factor=None, plain=None):
    """x_out [T, W] = x_in + y + add (y as for :func:`norm_step`, add [W] or None); h_t = sum_j conv[j] n_(t - taps + 1 + j) along every sequence
    with n = norm(x_out), conv [taps, W] fp32, state [slots, taps - 1, W] advanced.  Where nothing is added x_out may be None.
    ``factor`` [>= T * norm groups] fp32 scratch: the pass runs as two kernels, which steps of many rows gain from.  ``plain`` [T, ld] gets n."""
    t, w = x_in.shape
    if not x_in.is_cuda:
        new = reference.norm_step(x_in, y, None)
        if add is not None:
            new = new + add
        if x_out is not None:
            x_out.copy_(new)
        n = reference.rms(new, norm.w, norm.eps, norm.groups)
        if plain is not None:
            plain[:, :w] = n.to(plain.dtype)
        h[:, :w] = reference.short_conv(n, conv, state, si).to(h.dtype)
        return h
    src, ptrs, (k, ldy, lds, ldg, ldr), y_rows = _sublayer(y)
    assert plain is None or plain.dtype == h.dtype
    rc = _native.load().ogb_norm_conv_step(
        x_in.data_ptr(), _ptr(x_out), *ptrs, _ptr(add), norm.w.data_ptr(), conv.data_ptr(), state.data_ptr(), h.data_ptr(), _ptr(plain), _ptr(factor),
        float(norm.eps), t, w, norm.groups, conv.shape[0], k, x_in.stride(0), ldy, lds, ldg, ldr, h.stride(0), plain.stride(0) if plain is not None else 0, y_rows, *_rows_args(si, state), _ELEM[h.dtype], status_word().data_ptr(), _stream())
    _native.check(rc, "ogb_norm_conv_step")
    launch_counts["norm_conv_step"] += 1 if factor is None else 2
    return h


def _rows_args(si, state):
    return (si.ctx_len.data_ptr(), si.state_slot.data_ptr(), si.cu_q.data_ptr(), si.tile_seq.data_ptr(), si.tile_q0.data_ptr(), si.num_decode,
            si.num_tiles, state.shape[0])


@_timed("conv_rope_append")
def conv_rope_append(u, w, bias, state, q, pool, freq, si, nq, nk, nv, d, dv, dp, vp):
    """Short convolution over the projected rows u [T, nq d | nk d | nv dv] (w [taps, channels], bias added first, state
    [slots, taps - 1, channels] advanced), rotation of the first 2 len(freq) dimensions of every query and key (angles position x
    freq, fp64), queries to q [T, nq * dp], keys and values to the pages [nk][16][dp] | [nv][16][vp] of pool [pages, elements]."""
    if not u.is_cuda:
        reference.conv_rope_append(u, w, bias, state, q, pool, freq, si, nq, nk, nv, d, dv, dp, vp)
        return
    assert pool.dtype == u.dtype == q.dtype and freq.dtype == torch.float64
    rc = _native.load().ogb_conv_rope_append(
        u.data_ptr(), u.stride(0), w.data_ptr(), _ptr(bias), state.data_ptr(), w.shape[0], q.data_ptr(), q.stride(0), pool.data_ptr(), si.slots.data_ptr(),
        freq.data_ptr(), backed_pages(pool) * PAGE, pool.stride(0), nq, nk, nv, d, dv, dp, vp, 2 * freq.numel(), *_rows_args(si, state), _ELEM[u.dtype],
        status_word().data_ptr(), _stream())
    _native.check(rc, "ogb_conv_rope_append")
    launch_counts["conv_rope_append"] += 1


@_timed("conv_unit_gates")
def conv_unit_gates(u, w, state, ab, a_log, dt_bias, qk, v, gates, si, nk, nv, d, dv):
    """Short convolution and silu over the projected rows u [T, nk d | nk d | nv dv]; queries (times d^-1/2) and keys as unit vectors
    to qk [T, 2 nk d] fp32, values to v, and from ab [T, nv | nv] fp32 the log decay -exp(a_log) softplus(a + dt_bias) and the step size
    sigmoid(b) of every head to gates [T, nv, 2] fp32."""
    if not u.is_cuda:
        reference.conv_unit_gates(u, w, state, ab, a_log, dt_bias, qk, v, gates, si, nk, nv, d, dv)
        return
    assert qk.is_contiguous() and v.is_contiguous() and gates.is_contiguous() and v.dtype == u.dtype
    rc = _native.load().ogb_conv_unit_gates(
        u.data_ptr(), u.stride(0), w.data_ptr(), state.data_ptr(), w.shape[0], ab.data_ptr(), ab.stride(0), a_log.data_ptr(), dt_bias.data_ptr(),
        qk.data_ptr(), v.data_ptr(), gates.data_ptr(), nk, nv, d, dv, *_rows_args(si, state), _ELEM[u.dtype], status_word().data_ptr(), _stream())
    _native.check(rc, "ogb_conv_unit_gates")
    launch_counts["conv_unit_gates"] += 1


@_timed("delta_rule")
def delta_rule(qk, v, gates, state, out, heads, groups, dim, vdim, si, blocks=False, scratch=None):
    """Advance the gated delta rule over the step's rows (inputs of :func:`conv_unit_gates`): state [slots, heads, vdim,
    state_rows(dim)] fp32 in place, raw head outputs to out [T, heads * vdim] fp32.  ``blocks``: prompts in blocks of 64 tokens on
    the tensor cores, fp32 factors split in two tf32 terms; ``scratch(name, shape)`` provides fp32 scratch for them."""
    if not qk.is_cuda:
        reference.delta_rule(qk, v, gates, state, out, heads, groups, dim, vdim, si)
        return out
    assert out.is_contiguous()
    lib, work = _native.load(), None
    per_block = lib.ogb_delta_block_floats(heads, groups, dim, vdim) if blocks and si.num_prefill_seqs else 0
    if per_block:
        n = si.num_tiles * per_block
        work = scratch("delta_blocks", (n,)) if scratch is not None else torch.empty(n, dtype=torch.float32, device=qk.device)
    rc = lib.ogb_delta_rule(qk.data_ptr(), v.data_ptr(), gates.data_ptr(), state.data_ptr(), out.data_ptr(), heads, groups, dim, vdim,
                            si.ctx_len.data_ptr(), si.state_slot.data_ptr(), si.cu_q.data_ptr(), si.tile_seq.data_ptr(), si.tile_q0.data_ptr(),
                            si.num_decode, si.num_prefill_seqs, si.num_tiles, state.shape[0], _ptr(work), _ELEM[v.dtype], status_word().data_ptr(),
                            _stream())
    _native.check(rc, "ogb_delta_rule")
    launch_counts["delta_rule"] += 1
    return out


@_timed("diff_attention")
def diff_attention(q, out, pool, si, hq, hkv, d, dv, dp, vp, scale, lam, eps, gain, window=0, keep=0, splits=1, part_o=None, part_ml=None,
                   counters=None):
    """Differential attention: q [T, (head, map) dp], pages of :func:`conv_rope_append` (2 hkv key maps), out [T, hq * vp] =
    gain rms(a1 - lam a2).  ``window`` > 0: a query sees its last ``window`` keys and the first ``keep`` of the sequence."""
    if not q.is_cuda:
        reference.diff_attention(q, out, pool, si, hq, hkv, d, dv, dp, vp, scale, lam, eps, gain, window, keep)
        return out
    lib, st = _native.load(), status_word().data_ptr()
    nd, npf, t = si.num_decode, si.num_prefill_seqs, si.num_tokens
    tail = (si.page_table.shape[1], backed_pages(pool), pool.stride(0), hq, hkv, d, dv, dp, vp, q.stride(0), out.stride(0), int(window), int(keep),
            float(scale), float(lam), float(eps), float(gain))
    if nd > 0:
        rc = lib.ogb_diff_attention(q.data_ptr(), out.data_ptr(), pool.data_ptr(), si.page_table.data_ptr(), si.ctx_len.data_ptr(), 0, 0, 0, nd, 0, *tail,
                                    int(splits), _ptr(part_o), _ptr(part_ml), _ptr(counters), _ELEM[q.dtype], st, _stream())
        _native.check(rc, "ogb_diff_attention")
        launch_counts["diff_decode"] += 1
    if npf > 0:
        rc = lib.ogb_diff_attention(q[nd:].data_ptr(), out[nd:].data_ptr(), pool.data_ptr(), si.page_table[nd:].data_ptr(), si.ctx_len[nd:].data_ptr(),
                                    si.cu_q.data_ptr(), si.tile_seq.data_ptr(), si.tile_q0.data_ptr(), t - nd, si.num_tiles, *tail, 1, 0, 0, 0,
                                    _ELEM[q.dtype], st, _stream())
        _native.check(rc, "ogb_diff_attention")
        launch_counts["diff_prefill"] += 1
    return out


def set_diff_tc(on: bool) -> bool:
    """Switch the tensor-core kernels of differential attention (on by default); returns the old setting."""
    return bool(_native.load().ogb_diff_set_tc(int(on)))


@_timed("turn_table")
def turn_table(positions, freq, out):
    """Cosine and sine of position x freq (fp64 [n], angles reduced in double) to out [T, n, 2] fp32."""
    t = out.shape[0]
    if not out.is_cuda:
        reference.turn_table(positions[:t], freq, out)
        return out
    assert out.is_contiguous() and freq.dtype == torch.float64
    rc = _native.load().ogb_turn_table(positions.data_ptr(), freq.data_ptr(), out.data_ptr(), t, freq.numel(), _stream())
    _native.check(rc, "ogb_turn_table")
    launch_counts["turn_table"] += 1
    return out


@_timed("decay_memory")
def decay_memory(row, turns, logits, bias, cap, decay, state, peak, out, heads, dim, vdim, q_scale, k_scale, si, blocks=False, scratch=None):
    """Advance the matrix memories S <- a S + b k v^T of the step's rows and read o = S^T q out: row [T, ld] holds the projections
    [heads dim | heads dim | heads vdim] of q, k and v; q and k are rotated by ``turns`` (:func:`turn_table`; dimension i with i + n) where
    given, and scaled.  ``decay`` [2, heads] fp32 (decays, their logarithms): a = decay, b = 1.  Else ``logits`` [T, (input | forget) heads] fp32 plus
    ``bias``, capped at +-``cap``, are the gates of a memory with a running maximum (``peak`` [slots, heads]) and a normalizer (the state's
    last column), over which o is divided.  state [slots, heads, vdim (+ 1), state_rows(dim)] fp32 in place, out [T, heads * vdim] fp32.
    ``blocks``: prompts in blocks of 64 tokens on the tensor cores; ``scratch(name, shape)`` provides fp32 scratch for them."""
    if not row.is_cuda:
        reference.decay_memory(row, turns, logits, bias, cap, decay, state, peak, out, heads, dim, vdim, q_scale, k_scale, si)
        return out
    assert out.is_contiguous() and (logits is None) != (decay is None)
    lib, work = _native.load(), None
    per_block = lib.ogb_decay_block_floats(heads, dim, vdim, int(logits is not None)) if blocks and si.num_prefill_seqs else 0
    if per_block:
        n = si.num_tiles * per_block
        work = scratch("decay_blocks", (n,)) if scratch is not None else torch.empty(n, dtype=torch.float32, device=row.device)
    rc = lib.ogb_decay_memory(
        row.data_ptr(), row.stride(0), _ptr(turns), turns.shape[1] if turns is not None else 0, _ptr(logits), logits.stride(0) if logits is not None else 0,
        _ptr(bias), float(cap), _ptr(decay), state.data_ptr(), _ptr(peak), out.data_ptr(), heads, dim, vdim, state.shape[3], float(q_scale),
        float(k_scale), si.ctx_len.data_ptr(), si.state_slot.data_ptr(), si.cu_q.data_ptr(), si.tile_seq.data_ptr(), si.tile_q0.data_ptr(), si.num_decode,
        si.num_prefill_seqs, si.num_tiles, state.shape[0], _ptr(work), _ELEM[row.dtype], status_word().data_ptr(), _stream())
    _native.check(rc, "ogb_decay_memory")
    launch_counts["decay_memory"] += 1
    return out


def tied_page_elems(hkv, dp):
    """Elements of a page of keys that are values too: [hkv][16][dp] keys, and 16 fp32 factors (in room for two elements each)."""
    return hkv * PAGE * dp + 2 * PAGE


@_timed("tied_append")
def tied_append(row, q_bias, k_bias, q_gain, eps, factor, q, pool, slots, hq, hkv, d, dp):
    """Rows [T, hq d | hkv d] of projected queries and keys, biases added: queries over their root mean square (of the whole projection)
    times ``q_gain`` to q [T, hq * dp]; keys as they are to their slots of pool [pages, elements], with ``factor`` over their root mean
    square beside them -- the keys' norm and its weight reach a score through that number and the query's gain."""
    t = row.shape[0]
    if not row.is_cuda:
        reference.tied_append(row, q_bias, k_bias, q_gain, eps, factor, q, pool, slots, hq, hkv, d, dp)
        return
    assert pool.dtype == row.dtype == q.dtype
    rc = _native.load().ogb_tied_append(row.data_ptr(), row.stride(0), _ptr(q_bias), _ptr(k_bias), q_gain.data_ptr(), float(eps), float(factor), q.data_ptr(),
                                        q.stride(0), pool.data_ptr(), slots.data_ptr(), backed_pages(pool) * PAGE, pool.stride(0), t, hq, hkv, d, dp,
                                        _ELEM[row.dtype], status_word().data_ptr(), _stream())
    _native.check(rc, "ogb_tied_append")
    launch_counts["tied_append"] += 1


@_timed("tied_attention")
def tied_attention(q, out, pool, si, hq, hkv, d, dp, cap=0.0, slope=None, sink=None, window=0, gate=None, splits=1, part_o=None, part_ml=None,
                   counters=None):
    """Attention over pages of :func:`tied_append`, whose keys are the values: s = (q . k) factor, capped to cap tanh(s) where ``cap`` > 0
    (the factor then holds 1 / cap), less slope[head] x distance; softmax with exp(sink[head]) in the denominator; every head's output
    times the sigmoid of gate [T, hq].  ``window`` > 0: a query sees its last ``window`` keys.  slope, sink: fp32 [hq] or None."""
    if not q.is_cuda:
        reference.tied_attention(q, out, pool, si, hq, hkv, d, dp, cap, slope, sink, window, gate)
        return out
    lib, st = _native.load(), status_word().data_ptr()
    nd, npf, t = si.num_decode, si.num_prefill_seqs, si.num_tokens
    assert gate is None or gate.dtype == q.dtype
    tail = (si.page_table.shape[1], backed_pages(pool), pool.stride(0), hq, hkv, d, dp, q.stride(0), out.stride(0), gate.stride(0) if gate is not None else 0,
            int(window), float(cap))
    if nd > 0:
        rc = lib.ogb_tied_attention(q.data_ptr(), out.data_ptr(), pool.data_ptr(), si.page_table.data_ptr(), si.ctx_len.data_ptr(), 0, 0, 0, _ptr(gate),
                                    _ptr(slope), _ptr(sink), nd, 0, *tail, int(splits), _ptr(part_o), _ptr(part_ml), _ptr(counters), _ELEM[q.dtype], st,
                                    _stream())
        _native.check(rc, "ogb_tied_attention")
        launch_counts["tied_decode"] += 1
    if npf > 0:
        rc = lib.ogb_tied_attention(q[nd:].data_ptr(), out[nd:].data_ptr(), pool.data_ptr(), si.page_table[nd:].data_ptr(), si.ctx_len[nd:].data_ptr(),
                                    si.cu_q.data_ptr(), si.tile_seq.data_ptr(), si.tile_q0.data_ptr(), _ptr(gate[nd:] if gate is not None else None),
                                    _ptr(slope), _ptr(sink), t - nd, si.num_tiles, *tail, 1, 0, 0, 0, _ELEM[q.dtype], st, _stream())
        _native.check(rc, "ogb_tied_attention")
        launch_counts["tied_prefill"] += 1
    return out


def set_tied_tc(on: bool) -> bool:
    """Switch the tensor-core kernels of attention over keys that are values (on by default); returns the old setting."""
    return bool(_native.load().ogb_tied_set_tc(int(on)))
