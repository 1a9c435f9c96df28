"""Fizesun decoders (latent attention with a rotated part and head gates, looped layers, input convolutions, xIELU and clamped-gate
experts): every mechanism, the whole model and the serving path against the plain statement in oracle_fizesun.py, on the CPU path
and -- marked gpu -- on the kernels, in 32-bit and in bf16."""
import io
import json

import checkpoint_helpers
import numpy as np
import oracle_fizesun as O
import pytest
import torch
from checkpoint_helpers import CHUNKS, DEVICES, ENGINES, GPU, make_engine, replay_cuts, step_of, tokens_of, write_checkpoint

from onnx_genai_b200 import ops, replay
from onnx_genai_b200.engine.api import Engine, GenerateOptions
from onnx_genai_b200.models import hybrid, registry
from onnx_genai_b200.ops import hybrid as H
from onnx_genai_b200.ops import moe as M
from onnx_genai_b200.ops import reference

L, D, X = O.layer, O.ff_dense, O.ff_experts
# sizes that are no multiples of 8, a loop in the middle, a layer without a feed-forward, with and without a shared expert
MIXED = O.make_config(97, 72, [L(3, 20, 12, 28, 36, D(44)), L(4, 16, 6, 24, 44, X(6, 2, 24, shared=40)), L(2, 12, 10, 10, 18, None, scale=0.4),
                               L(5, 8, 4, 16, 24, X(5, 3, 35, limit=0.8), base=90.0)], loop=(1, 3, 3))
ODD = O.make_config(61, 50, [L(1, 10, 2, 14, 9, X(3, 1, 20, shared=9, shared_limit=0.6)), L(7, 6, 18, 5, 33, D(23), base=20000.0)], loop=(0, 1, 2), taps=1, eps=1e-2)
STRAIGHT = O.make_config(64, 64, [L(2, 16, 16, 16, 32, D(64)), L(2, 24, 8, 40, 16, D(32))], taps=5)
# shapes of the tensor-core kernels; the loop ends with the last layer
WIDE = O.make_config(80, 128, [L(4, 64, 32, 64, 128, X(4, 2, 64, shared=128)), L(2, 128, 64, 128, 256, D(256)), L(3, 32, 32, 48, 80, X(8, 3, 32))], loop=(1, 3, 2), taps=4)
ONCE = O.make_config(70, 68, [L(9, 7, 14, 9, 21, D(36)), L(2, 9, 6, 64, 70, D(20))], loop=(0, 2, 1), taps=2)
CONFIGS = {"mixed": MIXED, "odd": ODD, "straight": STRAIGHT, "wide": WIDE, "once": ONCE}
WHERE = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=GPU), pytest.param(("cuda", torch.bfloat16), marks=GPU)]


@pytest.fixture(scope="module")
def models():
    return {name: (cfg, O.random_tensors(cfg, seed=60 + i)) for i, (name, cfg) in enumerate(CONFIGS.items())}


def assert_logits(got, want, where):
    checkpoint_helpers.assert_logits(got, want, where, outliers=0.02)


def model_for(models, name, where):
    """In bf16 every expert is used, since rounding could tip a close choice (choosing is tested on fixed logits)."""
    cfg, tensors = models[name]
    if where[1] == "bf16":
        cfg, tensors = json.loads(json.dumps(cfg)), O.random_tensors(cfg, seed=80, sharp=1.0)
        for layer in cfg["layers"]:
            if layer["mlp"] and layer["mlp"]["kind"] == "moe":
                layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return cfg, tensors


def entries(si, order):
    """(sequence index, slot, first row, tokens before, rows) of a hand-made plan."""
    base, slots = 0, si.state_slot.cpu()
    for e, (a, n) in enumerate(order):
        yield e, int(slots[e]), base, a, n
        base += n


def up8(n):
    return n + (-n) % 8


def gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g)


# ------------------------------------------------------------------------------------------
# residual, norms, input convolutions
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("width,taps", [(40, 4), (37, 2), (72, 1), (1100, 3), (1030, 8), (2050, 4), (2048, 5), (4096, 4), (6000, 3)])
@pytest.mark.parametrize("kind", ["rows", "experts", "shared", "none"])
@pytest.mark.parametrize("halves", [False, True])
def test_norm_conv_step(where, width, taps, kind, halves):
    """x + output + vector, norm, and h + conv(h) along sequences that begin or go on, whose slots hold anything before they begin."""
    device, dt = where
    if halves and device == "cpu":
        pytest.skip("a variant of the CUDA kernels")
    r = gen(width + taps)
    si, order, _ = step_of(CHUNKS, device)
    t, eps, ld = si.num_tokens, 1e-3, up8(width)
    norm, filt = H.RmsNorm(torch.full((width,), 0.8), eps), r(width, taps) * 0.5
    past = [r(a, width) for a, _ in order]                # residual rows of earlier steps
    x, add = r(t, ld), r(width) if kind in ("rows", "experts") else None
    y, src = torch.zeros(t, width), None
    if kind == "rows":
        full = r(t, ld).to(dt)
        y, src = full[:, :width].float(), full.to(device)
    elif kind != "none":
        k = 3
        rows, pos, weight = r(t * k + 5, ld).to(dt), torch.randperm(t * k + 5)[:t * k].int().view(t, k), torch.rand(t, k)
        y = (rows[pos.long()].float() * weight[:, :, None]).sum(1)[:, :width]
        src = H.ExpertRows(rows.to(device), pos.to(device), weight.to(device))
        if kind == "shared":
            one, logits = r(t, ld).to(dt), r(t, 7)
            y = y + O.sigmoid(logits[:, 4:5]) * one[:, :width].float()
            src.shared, src.gate = one.to(device), logits.to(device)[:, 4]
    new = x[:, :width] + y + (add if add is not None else 0)
    state = torch.full((len(order), taps - 1, width), 9.0)
    for e, slot, _, a, _ in entries(si, order):
        h = O.rms(past[e], 0.8, eps)
        for k in range(min(a, taps - 1)):
            state[slot, taps - 2 - k] = h[a - 1 - k]
    state = state.to(device)
    h, xd = torch.zeros(t, ld, dtype=dt, device=device), x.to(device)
    x_out = torch.zeros(t, width, device=device) if kind != "none" else None
    if kind == "none":
        xd = xd[:, :width].contiguous()
    H.norm_conv_step(xd[:, :width], x_out, src, add.to(device) if add is not None else None, H.RmsNorm(norm.w.to(device), eps), hybrid.pack_input_conv(filt).to(device),
                     state, h, si, torch.zeros(t, device=device) if halves else None)
    if device == "cuda":
        ops.check_status()
    assert torch.equal(xd.cpu(), x[:, :xd.shape[1]]) and not h[:, width:].any()
    if x_out is not None:
        torch.testing.assert_close(x_out.cpu(), new, atol=2e-5, rtol=1e-5)
    tol = dict(atol=5e-5, rtol=1e-4) if dt == torch.float32 else dict(atol=0.02, rtol=0.01)
    for e, slot, b, a, n in entries(si, order):
        seq = O.rms(torch.cat([past[e], new[b:b + n]]), 0.8, eps)
        near = seq[max(0, a - taps):]
        want = O.sublayer_input(near, filt)[-n:]
        torch.testing.assert_close(h[b:b + n, :width].cpu().float(), want, **tol)
        if taps > 1:
            last = torch.cat([torch.zeros(taps, width), seq])[-(taps - 1):]
            live = min(a + n, taps - 1)
            torch.testing.assert_close(state[slot, taps - 1 - live:].cpu(), last[taps - 1 - live:], atol=5e-5, rtol=1e-5)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("width", [40, 37, 1100])
def test_norm_step_without_a_norm_behind(where, width):
    """x + y as it is, read out as it is or normed, for rows of the output too."""
    device, dt = where
    r = gen(width)
    ld = up8(width)
    x, y = r(9, width), r(9, ld).to(dt)
    want = x + y[:, :width].float()
    xd, both = x.clone().to(device), torch.zeros(9, 2 * ld, dtype=dt, device=device)
    pick, hl = torch.tensor([8, 0, 5], dtype=torch.int32, device=device), torch.zeros(3, ld, dtype=dt, device=device)
    norm = H.RmsNorm(torch.full((width,), 1.3, device=device), 1e-3)
    H.norm_step(xd, y.to(device), None, norm, hl, gather=pick)
    assert torch.equal(xd.cpu(), x)
    H.norm_step(xd, y.to(device), None, None, both[:, :width])
    torch.testing.assert_close(xd.cpu(), want, atol=1e-6, rtol=1e-6)
    assert torch.equal(both[:, :width].cpu(), xd.cpu().to(dt)) and not both[:, width:].any()
    tol = dict(atol=1e-5, rtol=1e-5) if dt == torch.float32 else dict(atol=0.02, rtol=0.01)
    torch.testing.assert_close(hl[:, :width].cpu().float(), O.rms(want, 1.3, 1e-3)[[8, 0, 5]], **tol)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("width", [40, 37, 1100])
def test_normed_embeddings_and_their_copy(where, width):
    device, dt = where
    table, ids = (gen(1)(13, width) * 3).to(dt), torch.tensor([12, 0, 7, 7], dtype=torch.int32)
    x, both = torch.zeros(4, 1, width, device=device), torch.zeros(4, 2 * up8(width), dtype=dt, device=device)
    H.embed_streams(ids.to(device), table.to(device), x, H.RmsNorm(torch.full((width,), 0.6, device=device), 1e-2), both[:, up8(width):up8(width) + width])
    want = O.rms(table[ids.long()].float(), 0.6, 1e-2)
    torch.testing.assert_close(x[:, 0].cpu(), want, atol=1e-5, rtol=1e-5)
    assert torch.equal(both[:, up8(width):up8(width) + width].cpu(), x[:, 0].cpu().to(dt)) and not both[:, :width].any()
    plain = torch.zeros(4, 1, width, device=device)
    H.embed_streams(ids.to(device), table.to(device), plain)
    assert torch.equal(plain[:, 0].cpu(), table[ids.long()].float())


# ------------------------------------------------------------------------------------------
# latent attention
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("heads,dim,rot,rank", [(3, 20, 12, 36), (1, 9, 2, 21), (16, 128, 64, 512), (5, 64, 66, 130)])
@pytest.mark.parametrize("split", [0, 4, 9])
def test_latents_rotations_and_their_places(where, heads, dim, rot, rank, split):
    """Normed latents and rotated key parts in their slots; query parts beside the folded queries below ``split``, in place behind."""
    device, dt = where
    r = gen(heads + rot)
    qw, cp, t, eps, base = up8(dim) + up8(rot), up8(rank), 9, 1e-3, 300.0
    row = r(t, heads * qw + cp + up8(rot) + 8).to(dt)
    w, slots = torch.rand(rank) + 0.5, torch.tensor([5, 16, 17, -1, 31, 0, 47, 33, 2], dtype=torch.int32)
    pos = torch.tensor([0, 1, 2, 3, 100, 4097, 65535, 1000003, 7], dtype=torch.int32)
    pool = torch.zeros(3, 16, cp + up8(rot), dtype=dt, device=device)
    q_out = torch.zeros(t * heads, cp + up8(rot), dtype=dt, device=device)
    got = row.clone().to(device)
    H.latent_append(got, heads * qw, w.to(device), eps, slots.to(device), pool, rank,
                    H.LatentRope(hybrid.rotation(rot, base, device), pos.to(device), heads, dim, q_out if split else None, cp, split))
    if device == "cuda":
        ops.check_status()
    tol = dict(atol=2e-6, rtol=1e-5) if dt == torch.float32 else dict(atol=0.02, rtol=0.01)
    turn = lambda x, p: O.rotate_pairs(x.double()[None], rot, base, start=int(p))[0].float()
    flat = pool.cpu().float().view(48, -1)
    part = heads * qw + cp
    for i, s in enumerate(slots.tolist()):
        if s >= 0:
            torch.testing.assert_close(flat[s, :rank], O.rms(row[i, heads * qw:heads * qw + rank].float(), w, eps), **tol)
            torch.testing.assert_close(flat[s, cp:cp + rot], turn(row[i, part:part + rot], pos[i]), **tol)
        for a in range(heads):
            c = a * qw + up8(dim)
            want = turn(row[i, c:c + rot], pos[i])
            mine = q_out[i * heads + a, cp:cp + rot] if i < split else got[i, c:c + rot]
            torch.testing.assert_close(mine.cpu().float(), want, **tol)
    unused = [s for s in range(48) if s not in slots.tolist()]
    assert not flat[unused].any() and not flat[:, cp + rot:].any() and not q_out[:, :cp].any() and not q_out[split * heads:].any()
    keep = torch.ones_like(row, dtype=torch.bool)
    for a in range(heads):
        keep[split:, a * qw + up8(dim):a * qw + up8(dim) + rot] = False
    assert torch.equal(got.cpu()[keep], row[keep])


def latent_case(where, heads, vrank, rot, chunks, spike, gated=True, splits=1, counters=None):
    """Attention over page rows [latent | rotated part]; ``spike``: position (from a sequence's length) of the one key that outshines
    the others -- in the rotated part for odd heads -- or None."""
    device, dt = where
    r = gen(heads * 100 + vrank + rot)
    width = up8(vrank) + up8(rot)
    si, order, pages = step_of(chunks, device, page_seed=5)
    t, table = si.num_tokens, si.page_table.cpu().long()
    pool, q = torch.zeros(pages, 16, width), torch.zeros(t, heads, width)
    q[..., :vrank], q[..., up8(vrank):up8(vrank) + rot] = r(t, heads, vrank), r(t, heads, rot)
    if spike is not None:
        q[:, 0::2, :vrank], q[:, 0::2, up8(vrank):] = 0.7 + 0.05 * q[:, 0::2, :vrank], 0.1 * q[:, 0::2, up8(vrank):]
        q[:, 1::2, :vrank] *= 0.1
        q[:, 1::2, up8(vrank):up8(vrank) + rot] = 0.7 + 0.05 * q[:, 1::2, up8(vrank):up8(vrank) + rot]
    rows = []
    for e, (a, n) in enumerate(order):
        c = torch.zeros(a + n, width)
        c[:, :vrank], c[:, up8(vrank):up8(vrank) + rot] = r(a + n, vrank) * 0.5, r(a + n, rot) * 0.5
        if spike is not None and 0 <= spike(a + n) < a + n:
            c[spike(a + n), :vrank] += 14.0 / vrank ** 0.5
            c[spike(a + n), up8(vrank):up8(vrank) + rot] += 14.0 / max(rot, 1) ** 0.5
        c = c.to(dt).float()
        j = torch.arange(a + n)
        pool[table[e, j // 16], j % 16] = c
        rows.append(c.double())
    q, gate = q.to(dt), r(t, heads + 3).to(dt)
    out = torch.zeros(t * heads, up8(vrank), dtype=dt, device=device)
    part_o, part_ml = torch.empty(t * heads * splits * up8(vrank), device=device), torch.empty(t * heads * splits * 2, device=device)
    scale = 1.4 * (vrank + rot) ** -0.5
    H.latent_attention(q.view(t * heads, width).to(device), out, pool.to(dt).to(device), si, heads, width, scale, 0, splits, part_o, part_ml, counters,
                       vrank=up8(vrank), gate=gate.to(device)[:, 2:2 + heads] if gated else None)
    if device == "cuda":
        ops.check_status()
    for e, _, b, a, n in entries(si, order):
        c = rows[e]
        seen = torch.arange(a + n)[None, :] <= torch.arange(a, a + n)[:, None]
        for h in range(heads):
            s = ((q[b:b + n, h].double() @ c.T) * scale).masked_fill(~seen, float("-inf"))
            want = torch.softmax(s, -1) @ c[:, :vrank] * (O.sigmoid(gate[b:b + n, 2 + h:3 + h].double()) if gated else 1)
            got = out.view(t, heads, -1)[b:b + n, h, :vrank].cpu().double()
            bound = (0.03 if dt == torch.bfloat16 else 3e-5) * max(1.0, float(want.abs().max()))
            assert (got - want).abs().max() < bound, (e, h, float((got - want).abs().max()))


# one size for every tile shape of the two tensor-core kernels, and one past them
LATENT_SIZES = [(3, 36, 12), (1, 18, 2), (6, 64, 16), (16, 104, 24), (5, 128, 64), (4, 184, 8), (20, 256, 64), (2, 320, 64), (3, 448, 64), (33, 512, 64), (2, 576, 32)]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("heads,vrank,rot", LATENT_SIZES)
def test_latent_attention_with_rotated_parts_and_gates(where, heads, vrank, rot):
    """Random keys, and one that stands out far away, at page borders, at the first token and at the query itself."""
    chunks = [(7, 1), (0, 1), (300, 1), (30, 2), (0, 2), (5, 17), (130, 70), (0, 150)]
    latent_case(where, heads, vrank, rot, chunks, None, gated=False)
    for spot in (lambda n: 0, lambda n: 1, lambda n: 16, lambda n: 15, lambda n: n - 1, lambda n: (n - 1) // 16 * 16, lambda n: n // 2):
        if where[0] == "cpu" and vrank > 200:
            break
        latent_case(where, heads, vrank, rot, chunks, spot)


@GPU
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,vrank,rot,splits", [(3, 36, 12, 4), (16, 104, 24, 3), (9, 128, 64, 5), (32, 256, 64, 8), (40, 512, 64, 6)])
def test_latent_decode_with_split_keys_and_gates(dtype, heads, vrank, rot, splits):
    chunks = [(7, 1), (0, 1), (400, 1), (255, 1), (15, 1), (16, 1), (299, 1), (1000, 1)]
    counters = torch.zeros(len(chunks) * -(-heads // 16), dtype=torch.int32, device="cuda")
    for c in (None, counters, counters):                  # merged by a second kernel, or by a row's last split (the counters come back as zeros)
        for spot in (None, lambda n: 3, lambda n: n - 1):
            latent_case(("cuda", dtype), heads, vrank, rot, chunks, spot, True, splits, c)
    assert (counters == 0).all()


EXPANDED = [(3, 20, 12, 28, 72), (2, 24, 40, 64, 96), (4, 64, 32, 64, 128), (2, 64, 64, 128, 200), (3, 128, 64, 128, 256), (2, 100, 60, 52, 512), (5, 33, 6, 17, 70)]


@GPU
@pytest.mark.parametrize("heads,dim,rot,vdim,rank", EXPANDED)
@pytest.mark.parametrize("spot", [None, 0, 15, 16, 77])
def test_prompts_on_expanded_keys_and_values(heads, dim, rot, vdim, rank, spot):
    """Keys and values expanded per head, with the rotated part behind every head's key, beside decoded rows that are left alone."""
    r, dt = gen(dim + rank), torch.bfloat16
    m = hybrid.LatentSpec(heads, dim, vdim, rank, 1.2 * (dim + rot) ** -0.5, rot_dim=rot, gated=True)
    assert hybrid.expand_prompts(m, dt)
    lin = lambda o, i: (r(o, i) / i ** 0.5).to(dt)
    uk, uv = lin(heads * dim, rank), lin(heads * vdim, rank)
    w = hybrid.pack_latent(m, lin(heads * (dim + rot), 64), lin(rank + rot, 64), torch.ones(rank), uk, uv, lin(64, heads * vdim), lin(heads, 64))
    si, order, pages = step_of([(7, 1), (0, 130), (30, 2), (100, 200), (65, 64), (0, 5)], "cuda", page_seed=2)
    t, table = si.num_tokens, si.page_table.cpu().long()
    q = torch.zeros(t, heads, m.q_width)
    q[..., :dim], q[..., up8(dim):up8(dim) + rot] = r(t, heads, dim), r(t, heads, rot)
    pool, rows = torch.zeros(pages, 16, m.key_width), []
    for e, (a, n) in enumerate(order):
        c = torch.zeros(a + n, m.key_width)
        c[:, :rank], c[:, up8(rank):up8(rank) + rot] = r(a + n, rank), r(a + n, rot)
        if spot is not None and spot < a + n:             # the shared part of one key outshines the others
            c[spot, up8(rank):up8(rank) + rot] = 12.0 / rot ** 0.5
            q[..., up8(dim):up8(dim) + rot] = 0.8 + 0.05 * q[..., up8(dim):up8(dim) + rot].clamp(-2, 2)
        c = c.to(dt).float()
        j = torch.arange(a + n)
        pool[table[e, j // 16], j % 16] = c
        rows.append(c.double())
    q, gate, vp = q.to(dt), r(t, heads).to(dt), up8(vdim)
    qc = torch.zeros(t, up8(m.proj_width), dtype=dt, device="cuda")
    qc[:, :heads * m.q_width], qc[:, m.gate_col:m.gate_col + heads] = q.view(t, -1).cuda(), gate.cuda()
    out = torch.full((t, heads * vp), 5.0, dtype=dt, device="cuda")
    n = H.visible_pages(si, 0)
    kc, vc = hybrid.chunks(m.q_width), hybrid.chunks(vdim)
    empty = lambda *s, dtype=dt: torch.full(s, 3.0, dtype=dtype, device="cuda")
    H.latent_prefill_expanded(qc, out, pool.to(dt).cuda(), w.kv.cuda(), si, heads, kc, vc, m.q_width, vp, m.scale, 0, n, empty(n * 16, m.key_width),
                              empty(n, heads, kc + vc, 16, 64), torch.zeros(si.num_prefill_seqs, si.page_table.shape[1], dtype=torch.int32, device="cuda"),
                              qc[:, m.gate_col:])
    ops.check_status()
    assert (out[:1] == 5.0).all()
    for e, _, b, a, k in entries(si, order):
        if k == 1:
            continue
        c = rows[e]
        keys, vals = (c[:, :rank] @ uk.double().T).view(-1, heads, dim), (c[:, :rank] @ uv.double().T).view(-1, heads, vdim)
        seen = torch.arange(a + k)[None, :] <= torch.arange(a, a + k)[:, None]
        for h in range(heads):
            qh = q[b:b + k, h].double()
            s = (qh[:, :dim] @ keys[:, h].T + qh[:, up8(dim):up8(dim) + rot] @ c[:, up8(rank):up8(rank) + rot].T) * m.scale
            want = torch.softmax(s.masked_fill(~seen, float("-inf")), -1) @ vals[:, h] * O.sigmoid(gate[b:b + k, h:h + 1].double())
            got = out[b:b + k, h * vp:h * vp + vdim].cpu().double()
            assert (got - want).abs().max() < 0.03 * max(1.0, float(want.abs().max())), (e, h, float((got - want).abs().max()))


# ------------------------------------------------------------------------------------------
# feed-forwards
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("m,ff,k", [(3, 40, 24), (1, 20, 72), (200, 96, 136), (70, 256, 128)])
def test_xielu_products(where, m, ff, k):
    device, dt = where
    r = gen(m)
    a, w = r(m, k).to(dt), (r(ff, k) * 3 / k ** 0.5).to(dt)
    if m > 1:
        a[0] = 0
    p, q = 0.7, -1.3
    layer = hybrid.HybridLayer(None, None, None)
    hybrid.pack_plain_mlp(layer, w, torch.zeros(8, ff, dtype=dt), hybrid.xielu(p, q))
    out = torch.full((m, up8(ff)), 7.0, dtype=dt, device=device)
    H.act_linear(a.to(device), layer.gate_up.to(device), layer.act, out)
    want = O.xielu(a.double() @ w.double().T, torch.tensor(p, dtype=torch.float64), torch.tensor(q, dtype=torch.float64))
    assert (out[:, :ff].cpu().double() - want).abs().max() < (1e-5 if dt == torch.float32 else 8e-3) * want.abs().max()
    assert not (m > 1 and out[0].any()) and not out[:, ff:].any()     # xIELU of nothing is nothing


def test_xielu_near_zero_and_far_out():
    z = torch.tensor([-60.0, -5.0, -1e-3, -1e-6, 0.0, 1e-6, 1e-3, 5.0, 60.0], dtype=torch.float64)
    for p, q in ((0.0, 0.0), (3.0, -4.0), (-30.0, 25.0)):
        act = hybrid.xielu(p, q)
        want = O.xielu(z, torch.tensor(p, dtype=torch.float64), torch.tensor(q, dtype=torch.float64))
        assert torch.isfinite(want).all()
        torch.testing.assert_close(reference.plain_act(z.float(), act).double(), want, atol=1e-6, rtol=1e-5)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("limit", [0.3, 2.0, 1e4])
def test_clamped_gate(where, limit):
    """Values inside and outside the limits: the gate is cut above only, the up value on both sides."""
    device, dt = where
    r = gen(8)
    for m, inter, k in ((3, 64, 40), (200, 40, 72), (70, 256, 128)):
        a, g, u = r(m, k).to(dt), (r(inter, k) * 3 / k ** 0.5).to(dt), (r(inter, k) * 3 / k ** 0.5).to(dt)
        packed, down, half = hybrid.pack_gated(g, u, r(8, inter).to(dt))
        n = down.shape[1]
        out = torch.zeros(m, n, dtype=dt, device=device)
        H.gated_linear(a.to(device), packed.to(device), half, H.Act("clamp_glu", limit), out, torch.zeros(m, 2 * n, dtype=dt, device=device))
        want = O.limited_expert(a.double(), g.double(), u.double(), torch.eye(inter, dtype=torch.float64), limit)
        assert (out[:, :inter].cpu().double() - want).abs().max() < (1e-5 if dt == torch.float32 else 8e-3) * want.abs().max()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("experts,top,hidden,inter,shared,tokens", [(6, 2, 40, 24, 0, 9), (8, 8, 72, 40, 56, 150), (5, 1, 20, 9, 33, 3), (64, 6, 128, 64, 128, 300),
                                                                     (4, 3, 264, 136, 20, 1), (256, 8, 64, 72, 8, 40)])
def test_clamped_experts_with_bias_and_a_shared_one(where, experts, top, hidden, inter, shared, tokens):
    device, dt = where
    r = gen(experts)
    lin = lambda o, i, s=1.0: (r(o, i) * s / i ** 0.5).to(dt)
    h = r(tokens, hidden).to(dt)
    W = {"router": lin(experts, hidden, 1.5), "router.b": r(experts) * 2, "shared.sg": lin(1, hidden, 2.0)}
    for e in range(experts):
        W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"] = lin(inter, hidden, 2.0), lin(inter, hidden, 2.0), lin(hidden, inter)
    if shared:
        W["shared.gate"], W["shared.up"], W["shared.down"] = lin(shared, hidden, 2.0), lin(shared, hidden, 2.0), lin(hidden, shared)
    part = lambda kind: [W[f"e{e}.{kind}"] for e in range(experts)]
    w = hybrid.pack_gated_moe(W["router"], W["router.b"], part("gate"), part("up"), part("down"),
                              tuple(W["shared." + n] for n in ("gate", "up", "down", "sg")) if shared else None)
    assert w.router.shape[0] == experts + (shared > 0)
    hp = torch.zeros(tokens, up8(hidden), dtype=dt)
    hp[:, :hidden] = h
    z = (h.double() @ W["router"].double().T).float()
    ws = M.MoEWorkspace(tokens, top, experts, up8(hidden), w.down.shape[2] + 8, device, dt, gated_f32=dt == torch.float32)   # as wide as a wider layer needs
    y = M.routed_experts(hp.to(device), z.to(device), w.up.to(device), w.down.to(device), ws, top, H.Act("clamp_glu", 1.1), w.half, renormalize=True,
                         bias=w.bias.to(device))
    if shared:
        mid, one = torch.zeros(tokens, w.shared_down.shape[1], dtype=dt, device=device), torch.zeros(tokens, up8(hidden), dtype=dt, device=device)
        H.gated_linear(hp.to(device), w.shared_up.to(device), w.shared_half, H.Act("clamp_glu", 0.7), mid,
                       torch.zeros(tokens, 2 * mid.shape[1], dtype=dt, device=device))
        H.linear(mid, w.shared_down.to(device), one[:, :hidden])
        y.shared, y.gate = one, (h.double() @ W["shared.sg"].double().T).float()[:, 0].to(device)
    x = torch.zeros(tokens, hidden, device=device)
    H.norm_step(x, y, None, None, None) if device == "cpu" else H.norm_step(x, y, None, None, torch.zeros(tokens, up8(hidden), dtype=dt, device=device))
    f = O.ff_experts(experts, top, inter, 1.1, shared, 0.7)
    want = O.experts(h.double(), {k: v.double() for k, v in W.items()}, f)
    assert (x.cpu().double() - want).abs().max() < (2e-5 if dt == torch.float32 else 0.02) * want.abs().max()


@pytest.mark.parametrize("device", DEVICES)
def test_chosen_experts_share_a_softmax_of_their_own(device):
    """Logits so far apart that most scores underflow still order the experts; the bias takes part in choice and weight."""
    if device == "cpu":
        ids, w = reference.moe_route(torch.tensor([[1.0, 2.0, 0.5, 3.0]]), 2, True, bias=torch.tensor([0.0, 4.0, 3.0, 0.0]))
        assert ids.tolist() == [[1, 2]] and torch.allclose(w[0], torch.softmax(torch.tensor([6.0, 3.5]), 0))
        return
    z = torch.tensor([[0.0, -150.0, -120.0, -300.0, -290.0, -1e4], [5.0, 4.0, 3.0, 2.0, 1.0, 0.0]], device="cuda")
    bias = torch.tensor([0.0, 0.0, 0.0, 0.0, -20.0, 30.0], device="cuda")
    ids, w = torch.zeros(2, 4, dtype=torch.int32, device="cuda"), torch.zeros(2, 4, device="cuda")
    lib = ops._native.load()
    assert lib.ogb_moe_route_grouped(z.data_ptr(), bias.data_ptr(), ids.data_ptr(), w.data_ptr(), 2, 6, 4, 1, 6, 1, 1, 0, 1, torch.cuda.current_stream().cuda_stream) == 0
    for t in range(2):
        want, ww = O.choose((z + bias)[t].cpu(), 4)
        assert ids[t].tolist() == want
        torch.testing.assert_close(w[t].cpu(), ww, atol=1e-6, rtol=1e-5)


# ------------------------------------------------------------------------------------------
# the whole model through the engine
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", ENGINES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_layer_runs(models, name, where):
    cfg, tensors = model_for(models, name, where)
    ids = tokens_of(cfg, 150, 1)
    layers = []
    want = O.forward(cfg, tensors, ids, layers_out=layers)
    eng = make_engine(cfg, tensors, where)
    assert eng.cfg.model.num_layers == len(O.layer_runs(cfg)) == len(eng.kv.pools) == len(eng.state.layers)
    eng.model.capture = []
    assert_logits(replay_cuts(eng, ids, [len(ids)]), want, where)
    assert len(eng.model.capture) == len(layers)
    for mine, ref in zip(eng.model.capture, layers):
        err = (mine[:150].cpu().double() - ref).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt()
        assert err < (0.04 if where[1] == "bf16" else 1e-5)


@pytest.mark.parametrize("where", ENGINES)
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("cuts", [[1], [2], [3, 1, 5, 2], [16], [17, 31, 1, 1, 64], [100, 1]])
def test_portions(models, name, where, cuts):
    cfg, tensors = model_for(models, name, where)
    ids = tokens_of(cfg, 118, 2)
    assert_logits(replay_cuts(make_engine(cfg, tensors, where), ids, cuts), O.forward(cfg, tensors, ids), where)


@pytest.mark.parametrize("where", ENGINES)
def test_unequal_requests_reuse_pages_and_slots(models, where):
    """Four live requests at most in a pool that holds no more than they need: portions beside decoded tokens, requests that
    pause, pages and slots handed on to the next request; every logits row as if alone."""
    cfg, tensors = model_for(models, "mixed", where)
    lengths = [100, 1, 37, 64, 90, 2, 16, 55, 33, 80]
    ids = {f"r{i}": tokens_of(cfg, n, 30 + i) for i, n in enumerate(lengths)}
    want = {k: O.forward(cfg, tensors, v) for k, v in ids.items()}
    rng = np.random.default_rng(4)
    eng = make_engine(cfg, tensors, where, max_tokens=320)
    rep, waiting, live, rows = replay.Replayer(eng), list(ids), {}, {k: [] for k in ids}
    while waiting or live:
        while waiting and len(live) < 4 and sum(-(-len(ids[k]) // 64) * 64 for k in [*live, waiting[0]]) <= 320:
            live[waiting.pop(0)] = 0
        batch, end = [], []
        for k in list(live):
            if rng.random() < 0.25 and len(live) > 1:
                continue
            n = min(int(rng.choice([1, 1, 2, 3, 7, 16, 30, 64])), len(ids[k]) - live[k])
            batch.append({"id": k, "tokens": ids[k][live[k]:live[k] + n], "want": list(range(n))})
            live[k] += n
            if live[k] == len(ids[k]):
                end.append(k)
                del live[k]
        out = rep.step(batch, end)
        for e in batch:
            rows[e["id"]] += [out.pop(0) for _ in e["want"]]
    for k in ids:
        assert_logits(torch.stack(rows[k]), want[k], where)
    assert eng.core.num_free_pages == eng.num_pages and eng.core.num_free_state_slots == 4


@GPU
def test_prompts_choose_between_latents_and_expansion(models):
    """Prompts with and without a past, beside decoded tokens: long ones on the expanded keys and values, short portions on the
    latents; the two agree."""
    where = ("cuda", "bf16")
    cfg, tensors = model_for(models, "wide", where)
    eng = make_engine(cfg, tensors, where, max_tokens=1664)
    ids = {k: tokens_of(cfg, 520, 90 + i) for i, k in enumerate("abc")}
    want = {k: O.forward(cfg, tensors, v) for k, v in ids.items()}
    rep, at, rows = replay.Replayer(eng), dict.fromkeys("abc", 0), {k: [] for k in "abc"}
    count = lambda: ops.launch_counts["latent_expand"]
    for portions, expanded in (({"a": 420}, True), ({"a": 1, "b": 450}, True), ({"a": 1, "b": 2, "c": 1}, False), ({"a": 1, "c": 519}, True), ({"a": 97, "b": 68}, False)):
        c0 = count()
        out = rep.step([{"id": k, "tokens": ids[k][at[k]:at[k] + n], "want": list(range(n))} for k, n in portions.items()], [])
        assert (count() > c0) == expanded
        for k, n in portions.items():
            rows[k] += [out.pop(0) for _ in range(n)]
            at[k] += n
    for k in "abc":
        assert_logits(torch.stack(rows[k]), want[k], where)


@pytest.mark.parametrize("where", ENGINES[:2])
@pytest.mark.parametrize("at", [0, 1, 2, 15, 16, 63, 100, 176, 178])
def test_single_tokens_show_in_logits(models, where, at):
    """Prompts that differ in one token -- the first ones, at page borders, far away, and just inside the input convolutions -- under
    sharpened attention; the oracle itself tells them apart by far more than the tolerance."""
    cfg, tensors = models["wide"]
    tensors = {k: v * 2 if k.endswith("mix.q") else v for k, v in tensors.items()}
    base = tokens_of(cfg, 180, 6)
    rows = []
    for tok in (3, 4):
        ids = list(base)
        ids[at] = tok
        want = O.forward(cfg, tensors, ids)
        assert_logits(replay_cuts(make_engine(cfg, tensors, where), ids, [50, 2, 60, 66, 1]), want, where)
        rows.append(want[-1])
    assert (rows[0] - rows[1]).pow(2).mean().sqrt() > 1e-3 * rows[0].std()


def test_mistakes_would_show(models, monkeypatch):
    """Mistakes planted in the oracle -- a pass's vector taken for another's, filters one tap off, gates, bias or norms left out, the
    activation's numbers swapped, other constants, halves rotated instead of neighbours -- move the logits by more than any tolerance."""
    cfg, tensors = models["mixed"]
    ids = tokens_of(cfg, 60, 3)
    want = O.forward(cfg, tensors, ids)
    spread = lambda got: float((got - want).pow(2).mean(-1).sqrt().max() / want.std())
    broken = {"step": {**tensors, "loop.step": tensors["loop.step"].flip(0)},
              "taps": {k: v.roll(1, 1) if "canon" in k else v for k, v in tensors.items()},
              "gate": {k: v * 0 if k.endswith("mix.g") else v for k, v in tensors.items()},
              "act": {k: v.flip(0) if k.endswith("mlp.act") else v for k, v in tensors.items()},
              "bias": {k: v * 0 if k.endswith("router.b") else v for k, v in tensors.items()},
              "norm": {**tensors, "embed.norm": tensors["embed.norm"] * 1.2}}
    for what, t in broken.items():
        assert spread(O.forward(cfg, t, ids)) > 0.02, what

    def other(*path, value):
        c = json.loads(json.dumps(cfg))
        at = c
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        return spread(O.forward(c, tensors, ids))

    assert other("loop", "times", value=2) > 0.02 and other("norm", "eps", value=0.1) > 1e-3
    for path, value in ((("mixer", "scale"), 0.1), (("mixer", "rot", "base"), 3.0)):
        assert other("layers", 0, *path, value=value) > 1e-3, path
    assert other("layers", 1, "mlp", "expert", "limit", value=0.5) > 1e-3 and other("layers", 1, "mlp", "shared", "limit", value=0.2) > 1e-3
    plain = O.rotate_pairs
    monkeypatch.setattr(O, "rotate_pairs", lambda x, dims, base, start=0: plain(x.view(len(x), 2, -1).transpose(1, 2).reshape(len(x), -1), dims, base, start))
    assert spread(O.forward(cfg, tensors, ids)) > 0.02


# ------------------------------------------------------------------------------------------
# serving: directory, scheduler, generation
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_in_batches(models, device, graphs, tmp_path):
    cfg, tensors = models["mixed"]
    d = write_checkpoint(tmp_path / "m", cfg, tensors)
    eng = Engine.from_dir(d, device=device, max_seqs=3, max_seq_len=300, num_pages=60, max_tokens_per_step=64, compute_dtype="f32",
                          cuda_graphs=graphs and device == "cuda")
    prompts = [tokens_of(cfg, n, 50 + n) for n in (5, 90, 1, 40, 17)]
    res = eng.generate_batch(prompts, GenerateOptions(max_new_tokens=24, greedy=True, ignore_eos=True))
    for p, r in zip(prompts, res):
        assert len(r.token_ids) == 24 and O.follows_greedily(cfg, tensors, p, r.token_ids)
    if graphs and device == "cuda":
        assert eng.llm.graph_replays > 0 and not eng.llm.graph_declines
    r = eng.generate(prompts[0], GenerateOptions(max_new_tokens=150, greedy=True, ignore_eos=True))      # long decoding
    assert len(r.token_ids) == 150 and O.follows_greedily(cfg, tensors, prompts[0], r.token_ids)


@GPU
def test_bf16_decoding_through_graphs_agrees_with_eager(models):
    cfg, tensors = models["wide"]
    outs = []
    for graphs in (False, True):
        eng = make_engine(cfg, tensors, ("cuda", "bf16"), max_tokens=1024, cuda_graphs=graphs, max_logit_rows=0)
        outs.append(eng.generate([tokens_of(cfg, n, 60 + n) for n in (5, 130, 40)], max_new_tokens=60, ignore_eos=True))
        assert not graphs or (eng.graph_replays > 0 and not eng.graph_declines)
    assert outs[0] == outs[1]


@pytest.mark.parametrize("device", DEVICES)
def test_preemption_recomputes_state(models, device):
    """A pool too small for all requests: victims lose pages and slot and are computed again, with the same tokens out."""
    cfg, tensors = models["once"]
    eng = make_engine(cfg, tensors, (device, "f32"), max_tokens=224, max_seqs=4, num_pages=14, max_tokens_per_step=64, prefill_chunk=64, max_logit_rows=0)
    prompts = [tokens_of(cfg, n, 70 + n) for n in (40, 50, 45)]
    outs = eng.generate(prompts, max_new_tokens=40, ignore_eos=True)
    assert eng.core.num_preemptions > 0
    for p, o in zip(prompts, outs):
        assert len(o) == 40 and O.follows_greedily(cfg, tensors, p, o)


@pytest.mark.parametrize("device", DEVICES)
def test_sampled_and_forced_requests_share_steps(models, device):
    cfg, tensors = models["odd"]
    eng = make_engine(cfg, tensors, (device, "f32"))
    ids, prompt = tokens_of(cfg, 40, 8), tokens_of(cfg, 12, 9)
    sid, hot = eng.add_request(prompt, 10, ignore_eos=True), eng.add_request(prompt, 10, temperature=0.8, top_k=20, seed=3, ignore_eos=True)
    fid, rows, out, at, drawn = eng.open_forced(ids[:15], [0, 14]), {}, [], 15, 0
    while len(out) < 10:
        step = eng.step()
        rows.update({p: r.cpu() for p, r in step.forced_logits.get(fid, [])})
        out += [t for s, t, _ in step.events if s == sid]
        drawn += sum(s == hot for s, _, _ in step.events)
        if at < 40:
            eng.extend_forced(fid, ids[at:at + 5], [4])
            at += 5
    assert O.follows_greedily(cfg, tensors, prompt, out) and drawn == 10
    assert_logits(torch.stack([rows[p] for p in sorted(rows)]), O.forward(cfg, tensors, ids)[sorted(rows)], (device, "f32"))
    eng.close_forced(fid)


def test_random_weights_of_the_family_run():
    """Seeded weights for benchmarks: every mechanism of the configuration is there."""
    read = registry.ARCHITECTURES["Fizesun"].read_config
    cfg = read(MIXED)
    w = registry.family_of(cfg).random_weights(cfg, "cpu", 1, 0, 0, torch.float32)
    assert w.loop_step.shape == (3, 72) and w.layers[1].moe.shared_up is not None and w.layers[3].moe.shared_up is None and w.layers[0].act.kind == "xielu"
    eng = replay.Replayer(checkpoint_helpers.LLMEngine(checkpoint_helpers.EngineConfig(model=cfg, num_pages=16, max_seqs=2, max_seq_len=64, compute_dtype="f32"), weights=w, device="cpu"))
    assert torch.isfinite(eng.step([{"id": "a", "tokens": [1, 2, 3], "want": [2]}], ["a"])[0]).all()
    per_layer = lambda i: 2 * (up8(cfg.layers[i].mixer.rank) + up8(cfg.layers[i].mixer.rot_dim))
    assert cfg.runs == [0, 1, 2, 1, 2, 1, 2, 3] and cfg.kv_bytes_per_token() == sum(per_layer(i) for i in cfg.runs) and cfg.weight_bytes() > 0


def test_configurations_that_cannot_run_are_refused(models):
    cfg, tensors = models["mixed"]
    read = registry.ARCHITECTURES["Fizesun"].read_config
    for path, value, what in ((("layers", 0, "type"), "other", "mixer type"), (("canon", "taps"), 9, "taps"), (("layers", 0, "mixer", "rot", "dims"), 6, "rotated"),
                              (("layers", 0, "mlp", "kind"), "other", "feed-forward"), (("layers", 1, "mlp", "router", "top"), 7, "cannot be chosen"),
                              (("loop", "stop"), 5, "loop"), (("loop", "times"), 0, "loop"), (("layers", 2, "mixer", "kv_rank"), 1100, "latent size")):
        bad = json.loads(json.dumps(cfg))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError, match=what):
            read(bad)
    c, load = read(cfg), registry.ARCHITECTURES["Fizesun"].load_weights
    assert load(c, {**tensors, "l9.extra": torch.zeros(1)}, torch.float32, "cpu").unused == ["l9.extra"]
    with pytest.raises(KeyError, match="l0.canon1"):
        load(c, {k: v for k, v in tensors.items() if k != "l0.canon1"}, torch.float32, "cpu")
    for kw, what in (({"max_draft_tokens": 2}, "speculative"), ({"kv_dtype": "fp8"}, "fp8")):
        with pytest.raises(ValueError, match=what):
            make_engine(cfg, tensors, ("cpu", "f32"), **{"compute_dtype": "bf16", **kw})


def test_directory_commands_and_replay(models, tmp_path, capsys):
    from onnx_genai_b200 import cli

    cfg, tensors = models["odd"]
    d = write_checkpoint(tmp_path / "m", cfg, tensors)
    assert cli.main(["show", d]) == 0
    assert json.loads(capsys.readouterr().out)["architecture"]["name"] == "Fizesun"
    assert cli.main(["validate", d]) == 0 and json.loads(capsys.readouterr().out)["ok"]
    prompt = tokens_of(cfg, 9, 4)
    rc = cli.main(["generate", d, "--device", "cpu", "--prompt-ids", ",".join(map(str, prompt)), "--greedy", "--max-new-tokens", "5"])
    out = [int(t) for t in capsys.readouterr().out.split()]
    assert rc == 0 and len(out) == 5 and O.follows_greedily(cfg, tensors, prompt, out)
    ids = tokens_of(cfg, 30, 5)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:20], "want": [3, 19]}, {"id": "b", "tokens": [1], "want": []}], "end": ["b"]},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[20:25], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": ids[25:], "want": [4]}], "end": ["a"]}]
    (tmp_path / "out").mkdir()
    said = []
    replay.serve(replay.build_engine(d, "float32", 128, "cpu"), str(tmp_path / "out"), io.StringIO("\n".join(map(json.dumps, lines))), said.append)
    assert said == ["done 0", "done 1", "done 2"]
    got = np.concatenate([np.fromfile(tmp_path / "out" / f"{s}.f32", dtype="<f4").reshape(-1, cfg["vocab"]) for s in (0, 2)])
    assert_logits(torch.from_numpy(got), O.forward(cfg, tensors, ids)[[3, 19, 29]], ("cpu", "f32"))
