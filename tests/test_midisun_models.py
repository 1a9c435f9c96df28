"""Midisun decoders (attention over keys that are the values, retention, mLSTM, sigmoid-routed experts in groups, norms in groups, gates
on the residual): every mechanism, the whole model and the serving path against the plain statement in oracle_midisun.py, on the CPU
path and -- marked gpu -- on the kernels, in 32-bit and in bf16."""
import io
import json

import checkpoint_helpers
import numpy as np
import oracle_midisun as O
import pytest
import torch
from checkpoint_helpers import CHUNKS, DEVICES, ENGINES, GPU, assert_logits, make_engine, replay_cuts, step_of, tokens_of, write_checkpoint

from onnx_genai_b200 import ops, replay
from onnx_genai_b200.engine.api import Engine, GenerateOptions
from onnx_genai_b200.models import hybrid, registry
from onnx_genai_b200.ops import hybrid as H
from onnx_genai_b200.ops import moe as M
from onnx_genai_b200.ops import reference

A, R, S, D, X = O.attention_layer, O.retention_layer, O.memory_layer, O.ff_dense, O.ff_experts
# sizes that are no multiples of 8, every mixer with every feed-forward, a layer without one
MIXED = O.make_config(97, 72, [A(6, 2, 20, 21, D(44), softcap=4.0), R(3, 20, 28, X(6, 2, 24, 3, 2), rot=12), S(2, 18, 30, None), S(4, 10, 6, X(8, 3, 35, 4, 3), cap=3.0),
                               R(2, 24, 10, D(20)), A(4, 4, 12, 50, X(5, 2, 16))], groups=3)
ODD = O.make_config(61, 50, [S(1, 9, 14, X(4, 1, 20, 2, 1)), R(5, 6, 18, D(23), base=20.0), A(3, 1, 10, 33, D(12), scale=0.9, softcap=1.5)], groups=5, taps=1, eps=1e-2, scale=2.5)
PLAIN = O.make_config(64, 64, [R(2, 32, 32, D(64)), R(4, 16, 16, D(32), rot=8, decay=[1.0, 0.5, 0.0, 0.9])], groups=1, taps=5, scale=1.0)
# shapes of the tensor-core kernels
WIDE = O.make_config(80, 128, [A(4, 2, 64, 70, D(128)), R(2, 64, 64, X(4, 2, 64, 2, 1)), S(2, 64, 128, X(8, 3, 32, 4, 2)), A(2, 1, 128, 130, D(64), softcap=9.0),
                               S(1, 128, 96, D(40)), R(1, 128, 160, D(40), rot=64)], groups=4, taps=4)
LONE = O.make_config(70, 68, [A(9, 9, 7, 1, D(36)), S(3, 16, 16, D(20), cap=30.0)], groups=2, taps=2)
CONFIGS = {"mixed": MIXED, "odd": ODD, "plain": PLAIN, "wide": WIDE, "lone": LONE}
WHERE = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=GPU), pytest.param(("cuda", torch.bfloat16), marks=GPU)]


@pytest.fixture(scope="module")
def models():
    return {name: (cfg, O.random_tensors(cfg, seed=90 + i)) for i, (name, cfg) in enumerate(CONFIGS.items())}


def model_for(models, name, where):
    """In bf16 every expert is used, since rounding could tip a close choice (choosing is tested on fixed logits); the norms' eps keeps head
    outputs that are next to nothing -- one query that hardly meets one key -- from being magnified with their rounding, and input gates
    are low, so that no read-out is divided by a normalizer that happens to vanish."""
    cfg, tensors = models[name]
    if where[1] == "bf16":
        cfg, tensors = json.loads(json.dumps(cfg)), O.random_tensors(cfg, seed=110, sharp=1.0)
        cfg["norm"]["eps"] = 0.05
        tensors = {k: v - 3 if k.endswith("mix.i.b") else v / 4 if k.endswith("mix.i") else v for k, v in tensors.items()}
        for layer in cfg["layers"]:
            if layer["mlp"] and layer["mlp"]["kind"] == "moe":
                r = layer["mlp"]["router"]
                r["top"], r["groups"]["keep"] = r["experts"], r["groups"]["count"]
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


def to(device, *ts):
    return [None if t is None else t.to(device) for t in ts]


# ------------------------------------------------------------------------------------------
# residual: norms in groups, gates, input convolutions, embeddings
# ------------------------------------------------------------------------------------------
def sublayer_output(r, kind, t, ld, width, dt, device):
    """(what a sublayer leaves, on the device; its sum) for rows or expert rows."""
    if kind == "rows":
        full = r(t, ld).to(dt)
        return full.to(device), full[:, :width].float()
    k = 3
    rows, pos, weight = r(t * k + 5, ld).to(dt), torch.randperm(t * k + 5)[:t * k].int().view(t, k), torch.rand(t, k)
    return H.ExpertRows(*to(device, rows, pos, weight)), (rows[pos.long()].float() * weight[:, :, None]).sum(1)[:, :width]


RESIDUAL = [(40, 4, 1), (36, 3, 4), (50, 1, 5), (72, 5, 3), (1100, 3, 11), (1030, 2, 2), (2048, 4, 4), (4096, 3, 8), (6000, 2, 3), (64, 4, 64)]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("width,taps,groups", RESIDUAL)
@pytest.mark.parametrize("kind", ["rows", "experts"])
@pytest.mark.parametrize("halves", [False, True])
def test_gated_residual_norm_in_groups_and_input_convolution(where, width, taps, groups, kind, halves):
    """x + (output + bias) sigmoid(gate), its norm in groups, and h + conv(h), along sequences that begin or go on."""
    device, dt = where
    if halves and device == "cpu":
        pytest.skip("a variant of the CUDA kernels")
    r = gen(width + taps)
    si, order, _ = step_of(CHUNKS, device)
    t, eps, ld = si.num_tokens, 1e-3, up8(width)
    gain, filt, past = 0.5 + torch.rand(width), r(width, taps) * 0.5, [r(a, width) for a, _ in order]
    src, y = sublayer_output(r, kind, t, ld, width, dt, device)
    x, gate, gate_bias, bias = r(t, width), (2 * r(t, ld)).to(dt), r(width), r(width) if kind == "rows" else None
    new = x + (y + (bias if bias is not None else 0)) * O.sigmoid(gate[:, :width].float() + gate_bias)
    state = torch.full((len(order), taps - 1, width), 9.0)
    for e, slot, _, a, _ in entries(si, order):
        h = O.rms_in_groups(past[e], gain, groups, eps)
        for k in range(min(a, taps - 1)):
            state[slot, taps - 2 - k] = h[a - 1 - k]
    state = state.to(device)
    h, plain, xd, x_out = torch.zeros(t, ld, dtype=dt, device=device), torch.zeros(t, ld, dtype=dt, device=device), x.to(device), torch.zeros(t, width, device=device)
    gated = H.GatedRows(src, *to(device, gate, gate_bias, bias))
    norm = H.RmsNorm(gain.to(device), eps, groups)
    H.norm_conv_step(xd, x_out, gated, None, norm, hybrid.pack_input_conv(filt).to(device), state, h, si,
                     torch.zeros(t * groups, device=device) if halves else None, plain)
    if device == "cuda":
        ops.check_status()
    assert torch.equal(xd.cpu(), x) and not h[:, width:].any() and not plain[:, width:].any()
    torch.testing.assert_close(x_out.cpu(), new, atol=2e-5, rtol=1e-5)
    tol = dict(atol=5e-5, rtol=1e-4) if dt == torch.float32 else dict(atol=0.02, rtol=0.01)
    torch.testing.assert_close(plain[:, :width].cpu().float(), O.rms_in_groups(new, gain, groups, eps), **tol)
    for e, slot, b, a, n in entries(si, order):
        seq = O.rms_in_groups(torch.cat([past[e], new[b:b + n]]), gain, groups, eps)
        torch.testing.assert_close(h[b:b + n, :width].cpu().float(), O.sublayer_input(seq[max(0, a - taps):], filt)[-n:], **tol)
        if taps > 1:
            last, live = torch.cat([torch.zeros(taps, width), seq])[-(taps - 1):], min(a + n, taps - 1)
            torch.testing.assert_close(state[slot, taps - 1 - live:].cpu(), last[taps - 1 - live:], atol=5e-5, rtol=1e-5)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("width,groups", [(40, 1), (36, 4), (50, 5), (1030, 2), (4096, 4), (9000, 3), (12288, 8)])
@pytest.mark.parametrize("kind", ["rows", "experts"])
def test_gated_residual_in_place_and_gathered(where, width, groups, kind):
    device, dt = where
    r, t, eps, ld = gen(width), 37, 1e-2, up8(width)
    src, y = sublayer_output(r, kind, t, ld, width, dt, device)
    x, gain, gate, gate_bias = r(t, width), 0.5 + torch.rand(width), r(t, ld).to(dt), r(width)
    new = x + y * O.sigmoid(gate[:, :width].float() + gate_bias)
    want = O.rms_in_groups(new, gain, groups, eps)
    gated, norm = H.GatedRows(src, *to(device, gate, gate_bias)), H.RmsNorm(gain.to(device), eps, groups)
    tol = dict(atol=3e-5, rtol=1e-4) if dt == torch.float32 else dict(atol=0.02, rtol=0.01)
    xd, at = x.to(device), torch.tensor([36, 0, 5], dtype=torch.int32)
    few = torch.zeros(3, ld, dtype=dt, device=device)
    H.norm_step(xd, gated, None, norm, few, at.to(device))
    assert torch.equal(xd.cpu(), x)                       # gathered rows leave the residual alone
    torch.testing.assert_close(few[:, :width].cpu().float(), want[at.long()], **tol)
    h = torch.zeros(t, ld, dtype=dt, device=device)
    H.norm_step(xd, gated, None, norm, h)
    torch.testing.assert_close(xd.cpu(), new, atol=2e-5, rtol=1e-5)
    torch.testing.assert_close(h[:, :width].cpu().float(), want, **tol)
    if device == "cuda":
        ops.check_status()


@pytest.mark.parametrize("where", WHERE)
def test_scaled_embeddings(where):
    device, dt = where
    table, ids = torch.randn(30, 44).to(dt), torch.tensor([3, 29, 0, 3], dtype=torch.int32)
    x = torch.zeros(4, 1, 44, device=device)
    H.embed_streams(ids.to(device), table.to(device), x, scale=0.3)
    torch.testing.assert_close(x[:, 0].cpu(), table[ids.long()].float() * 0.3)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("heads,n", [(3, 128), (2, 256), (5, 20), (1, 70)])
@pytest.mark.parametrize("weight", ["none", "shared", "heads"])
@pytest.mark.parametrize("act", ["silu", "sigmoid"])
def test_head_norms_and_gates(where, heads, n, weight, act):
    device, dt = where
    r = gen(n)
    x, gate = r(9, heads * n + 3), r(9, up8(heads * n)).to(dt)
    w = {"none": None, "shared": r(n), "heads": r(heads * n)}[weight]
    out = torch.zeros(9, up8(heads * n), dtype=dt, device=device)
    H.head_rmsnorm(x.to(device), None if w is None else w.to(device), 1e-2, out, heads, n, gate=gate.to(device)[:, :heads * n], gate_act=act)
    y = O.rms(x[:, :heads * n].view(9, heads, n), 1.0, 1e-2)
    y = (y * (1 if w is None else w if weight == "shared" else w.view(heads, n))).flatten(1) * (O.silu if act == "silu" else O.sigmoid)(gate[:, :heads * n].float())
    torch.testing.assert_close(out[:, :heads * n].cpu().float(), y, **(dict(atol=2e-5, rtol=1e-5) if dt == torch.float32 else dict(atol=0.03, rtol=0.01)))


# ------------------------------------------------------------------------------------------
# routing
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", WHERE[:2])
@pytest.mark.parametrize("count,top,groups,keep", [(6, 2, 3, 2), (8, 3, 4, 3), (8, 4, 2, 1), (5, 2, 1, 1), (6, 4, 6, 4), (64, 6, 8, 3), (256, 8, 16, 4), (33, 32, 1, 1), (4, 4, 2, 2)])
def test_sigmoid_routing_with_corrected_choice(where, count, top, groups, keep):
    """Choices by corrected scores, groups by the sum of their two best, weights without the correction; all corrections may be negative."""
    device, _ = where
    r = gen(count)
    for shift in (0.0, -3.0):
        z, corr = r(40, count) * 3, r(count) * 0.6 + shift
        ids, w = reference.moe_route(z, top, True, groups, keep, corr, "sigmoid", 2)
        if device == "cuda":
            dev_ids, dev_w = torch.zeros(40, top, dtype=torch.int32, device=device), torch.zeros(40, top, device=device)
            zc, cc = z.to(device), corr.to(device)
            rc = ops._native.load().ogb_moe_route_grouped(zc.data_ptr(), cc.data_ptr(), dev_ids.data_ptr(), dev_w.data_ptr(), 40, count, top, 1, count, groups, keep, 1, 2,
                                                          torch.cuda.current_stream().cuda_stream)
            assert rc == 0
            ids, w = dev_ids.cpu(), dev_w.cpu()
        for t in range(40):
            want, share = O.choose(z[t].double(), corr.double(), top, groups, keep)
            mine = dict(zip(ids[t].tolist(), w[t].tolist()))
            assert sorted(mine) == sorted(want)
            for e, s in zip(want, share):
                assert abs(mine[e] - float(s)) < 1e-6


def test_group_scores_are_sums_of_two():
    """A group with two good experts beats one with the single best; the other rule would choose differently."""
    z = torch.logit(torch.tensor([[0.9, 0.05, 0.6, 0.55]]))
    assert sorted(reference.moe_route(z, 2, True, 2, 1, torch.zeros(4), "sigmoid", 2)[0][0].tolist()) == [2, 3]
    assert sorted(reference.moe_route(z, 2, True, 2, 1, torch.zeros(4), "sigmoid", 1)[0][0].tolist()) == [0, 1]
    ids, w = reference.moe_route(z, 1, True, 2, 1, torch.tensor([-2.0, 0, 0, 0]), "sigmoid", 2)
    assert ids[0].tolist() == [2] and w[0].tolist() == [1.0]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("hidden,ff,count,top,groups,keep,t", [(40, 24, 6, 2, 3, 2, 9), (72, 35, 8, 3, 4, 3, 150), (128, 64, 16, 4, 4, 2, 300)])
def test_routed_silu_experts(where, hidden, ff, count, top, groups, keep, t):
    device, dt = where
    r, up = gen(hidden), up8(hidden)
    h, z, corr = r(t, hidden).to(dt), r(t, count) * 2, r(count) * 0.3
    W = {f"e{e}.{k}": (r(*((ff, hidden) if k != "down" else (hidden, ff))) / hidden ** 0.5).to(dt) for e in range(count) for k in ("gate", "up", "down")}
    w = hybrid.pack_gated_moe(r(count, hidden), corr, *([W[f"e{e}.{k}"].to(device) for e in range(count)] for k in ("gate", "up", "down")))
    ws = M.MoEWorkspace(t, top, count, up, w.down.shape[2], device, dt, gated_f32=dt == torch.float32)
    hp = torch.zeros(t, up, dtype=dt)
    hp[:, :hidden] = h
    y = M.routed_experts(hp.to(device), z.to(device), w.up, w.down, ws, top, "silu", w.half, groups, keep, True, corr.to(device), "sigmoid", 2)
    got = (y.rows[y.pos.long()].float() * y.weight[:, :, None]).sum(1)[:, :hidden].cpu()
    want = torch.zeros(t, hidden)
    for i in range(t):
        for e, s in zip(*O.choose(z[i], corr, top, groups, keep)):
            want[i] += s * O.gated(h[i].float(), *(W[f"e{e}.{k}"].float() for k in ("gate", "up", "down")))
    assert (got - want).abs().max() < (2e-5 if dt == torch.float32 else 0.03) * want.abs().max()


# ------------------------------------------------------------------------------------------
# attention over keys that are the values
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("hq,hkv,d", [(6, 2, 20), (4, 4, 64), (1, 1, 9), (16, 2, 128), (3, 1, 300)])
@pytest.mark.parametrize("biased", [False, True])
def test_projections_reach_queries_and_pages(where, hq, hkv, d, biased):
    """Biases, norms over whole projections, and pages: what a query and a page say together is the score."""
    device, dt = where
    r, dp, eps, factor = gen(d), up8(d), 1e-2, 0.37
    si, order, pages = step_of([(3, 1), (0, 2), (9, 30)], device)
    t = si.num_tokens
    row = r(t, (hq + hkv) * d + 5).to(dt)
    qb, kb = (r(hq * d), r(hkv * d)) if biased else (None, None)
    qn, kn = r(hq * d), r(hkv * d)
    spec = hybrid.TiedSpec(hq, hkv, d, 1.0, gated=False)
    w = hybrid.pack_tied(spec, torch.zeros(hq * d, 8), torch.zeros(hkv * d, 8), None, qb, kb, qn, kn, None, None, torch.zeros(8, hq * d), None)
    pool = torch.full((pages, H.tied_page_elems(hkv, dp)), 5.0, dtype=dt, device=device)
    q = torch.full((t, hq * dp), 5.0, dtype=dt, device=device)
    slots = si.slots.clone()
    slots[1] = -1                                          # a padding row writes nothing
    H.tied_append(row.to(device), *to(device, w.q_bias, w.k_bias, w.q_gain), eps, factor, q, pool, slots, hq, hkv, d, dp)
    if device == "cuda":
        ops.check_status()
    keys, factors = reference.tied_pages(pool.cpu(), hkv, dp)
    qs = row[:, :hq * d].float() + (qb if biased else 0)
    ks = row[:, hq * d:(hq + hkv) * d].float() + (kb if biased else 0)
    tol = dict(atol=2e-5, rtol=1e-4) if dt == torch.float32 else dict(atol=0.05, rtol=0.02)
    nq, nk = O.rms(qs, qn, eps).view(t, hq, d), O.rms(ks, kn, eps).view(t, hkv, d).repeat_interleave(hq // hkv, 1)
    for i in range(t):
        slot = int(slots[i])
        if slot < 0:
            assert (keys[int(si.slots[i]) // 16, :, int(si.slots[i]) % 16] == 5).all()
            continue
        k = keys[slot // 16, :, slot % 16]
        torch.testing.assert_close(k[:, :d].float(), ks[i].view(hkv, d), **tol)
        got = torch.einsum("hd,hd->h", q[i].cpu().float().view(hq, dp), k.float().repeat_interleave(hq // hkv, 0)) * factors[slot // 16, slot % 16]
        torch.testing.assert_close(got, (nq[i] * nk[i]).sum(-1) * factor, atol=1e-4 if dt == torch.float32 else 0.03 * d ** 0.5, rtol=1e-3)


def tied_case(where, hq, hkv, d, window, cap, chunks, spike, sloped=True, splits=1, counters=None):
    """Attention over random pages; ``spike``: a key that outshines the others, at a position of the sequence."""
    device, dt = where
    r = gen(hq * 1000 + d)
    si, order, pages = step_of(chunks, device, page_seed=3)
    dp, t = up8(d), si.num_tokens
    pool = torch.zeros(pages, H.tied_page_elems(hkv, dp), dtype=dt)
    keys, factors = reference.tied_pages(pool, hkv, dp)
    table, kv = si.page_table.cpu().long(), []
    q = r(t, hq, d) if spike is None else 0.7 + 0.05 * r(t, hq, d)
    for e, (a, n) in enumerate(order):
        k, f = r(a + n, hkv, d) * (1.0 if spike is None else 0.3), (0.6 + 0.8 * torch.rand(a + n)) * d ** -0.5
        at = spike(a + n) if spike is not None else -1
        if 0 <= at < a + n:
            k[at], f[at] = 1.0, 9.0 / (0.7 * d)
        if cap > 0:
            f = f / cap
        k, j = k.to(dt), torch.arange(a + n)
        keys[table[e, j // 16], :, j % 16, :d] = k
        factors[table[e, j // 16], j % 16] = f
        kv.append((k.double(), f.double()))
    if window > 0:                                        # pages that no query sees are gone
        for e, (a, n) in enumerate(order):
            si.page_table[e, :max(0, (a - window + 1) // 16)] = -1
    slope = 2.0 ** -torch.arange(2, hq + 2).float().clamp(max=9) if sloped else None
    sink, gate, q = r(hq) + 1, r(t, hq + 3).to(dt), q.to(dt)
    qp = torch.zeros(t, hq, dp, dtype=dt)
    qp[..., :d] = q
    out = torch.full((t, hq * dp), 3.0, dtype=dt, device=device)
    units = hkv * -(-(hq // hkv) // 16)
    part_o, part_ml = torch.empty(t * units * 16 * splits * dp, device=device), torch.empty(t * units * 32 * splits, device=device)
    H.tied_attention(qp.view(t, -1).to(device), out, pool.to(device), si, hq, hkv, d, dp, cap, *to(device, slope, sink), window, gate.to(device)[:, :hq], splits,
                     part_o, part_ml, counters)
    if device == "cuda":
        ops.check_status()
    for e, slot, b, a, n in entries(si, order):
        k, f = kv[e]
        i = torch.arange(a, a + n)
        dist = i[:, None] - torch.arange(a + n)[None, :]
        for h in range(hq):
            c = h // (hq // hkv)
            s = q[b:b + n, h].double() @ k[:, c].T * f
            s = cap * torch.tanh(s) if cap > 0 else s
            s = s - (float(slope[h]) if sloped else 0.0) * dist
            p = torch.exp(s.masked_fill((dist < 0) | ((dist >= window) if window > 0 else False), float("-inf")))
            want = (p @ k[:, c]) / (p.sum(-1, keepdim=True) + torch.exp(sink[h].double())) * O.sigmoid(gate[b:b + n, h:h + 1].double())
            got = out[b:b + n, h * dp:h * dp + d].cpu().double()
            assert (got - want).abs().max() < (0.02 if dt == torch.bfloat16 else 3e-5), (e, h, int((got - want).abs().amax(1).argmax()))
    assert not out.view(t, hq, dp)[..., d:].any()


TIED_SIZES = [(3, 1, 20, 21, 4.0), (1, 1, 10, 1, 0.0), (4, 2, 64, 70, 6.0), (8, 1, 32, 100, 3.0), (20, 1, 48, 64, 30.0), (2, 2, 128, 130, 5.0), (3, 3, 104, 90, 20.0),
              (2, 1, 160, 40, 8.0), (2, 2, 256, 30, 0.0), (6, 3, 64, 0, 2.0), (1, 1, 300, 33, 7.0), (66, 1, 16, 50, 5.0)]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("hq,hkv,d,window,cap", TIED_SIZES)
def test_attention_edges(where, hq, hkv, d, window, cap):
    """Random keys, and keys that stand out just inside and just outside the window, at the first tokens, at page borders and far away."""
    chunks = [(7, 1), (0, 1), (window + 40, 1), (300, 1), (30, 2), (0, 2), (5, 17), (210, 70), (0, 150), (250, 3)]
    tied_case(where, hq, hkv, d, window, cap, chunks, None)
    spots = [lambda n: 0, lambda n: 1, lambda n: 15, lambda n: 16, lambda n: n - 1, lambda n: n - 2]
    if window > 0:
        spots += [lambda n: n - window, lambda n: n - 1 - window, lambda n: n - window + 1]
    for spot in spots:
        tied_case(where, hq, hkv, d, window, cap, chunks, spot, sloped=False)


@GPU
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hq,hkv,d,window,cap,splits", [(3, 1, 24, 0, 4.0, 4), (8, 2, 64, 300, 0.0, 3), (4, 4, 128, 200, 20.0, 8), (18, 1, 64, 0, 3.0, 5), (32, 2, 256, 0, 6.0, 2)])
def test_decode_with_split_keys(dtype, hq, hkv, d, window, cap, splits):
    chunks = [(7, 1), (0, 1), (400, 1), (255, 1), (15, 1), (16, 1), (299, 1), (300, 1), (900, 1)]
    counters = torch.zeros(len(chunks) * hq, dtype=torch.int32, device="cuda")
    for spot in (None, (lambda n: n - window) if window else (lambda n: 20), lambda n: 1):
        for _ in range(2):                                # the counters come back as zeros
            tied_case(("cuda", dtype), hq, hkv, d, window, cap, chunks, spot, spot is None, splits, counters)
    assert (counters == 0).all()


@pytest.mark.parametrize("where", WHERE)
def test_scores_far_above_the_cap_and_sinks_that_take_all(where):
    """Scores of hundreds, all capped alike; sinks above and below every score; the softmax of either is finite."""
    device, dt = where
    chunks, hq, d = [(40, 1), (0, 130)], 4, 64
    si, order, pages = step_of(chunks, device)
    pool = torch.zeros(pages, H.tied_page_elems(1, d), dtype=dt)
    keys, factors = reference.tied_pages(pool, 1, d)
    keys[:], factors[:] = 1.0, 100.0
    q = torch.full((si.num_tokens, hq * d), 1.0, dtype=dt, device=device)
    sink = torch.tensor([500.0, -500.0, 20.0, float("-inf")])
    out = torch.zeros(si.num_tokens, hq * d, dtype=dt, device=device)
    H.tied_attention(q, out, pool.to(device), si, hq, 1, d, d, 20.0, None, sink.to(device), 0)
    n = torch.tensor([a + i + 1 for a, m in order for i in range(m)]).float()
    want = torch.stack([torch.zeros_like(n), torch.ones_like(n), n / (n + 1), torch.ones_like(n)], 1)
    torch.testing.assert_close(out.view(-1, hq, d).cpu().float(), want[:, :, None].expand(-1, -1, d), atol=5e-3 if dt == torch.bfloat16 else 1e-5, rtol=1e-3)


# ------------------------------------------------------------------------------------------
# matrix memories
# ------------------------------------------------------------------------------------------
def memory_after(q, k, v, i, f, decay):
    """(read-outs, state, normalizer, maximum) of one head after its tokens."""
    if decay is not None:
        rows, state = O.retention_head(q, k, v, decay), torch.zeros(k.shape[1], v.shape[1], dtype=k.dtype)
        for t in range(len(k)):
            state = decay * state + torch.outer(k[t], v[t])
        return rows, state, None, None
    rows = O.matrix_memory_head(q, k, v, i, f) if len(q) else q
    state, norm, m = torch.zeros(k.shape[1], v.shape[1], dtype=k.dtype), torch.zeros(k.shape[1], dtype=k.dtype), 0.0
    for t in range(len(k)):
        new = max(float(f[t]) + m, float(i[t]))
        a, b = np.exp(float(f[t]) + m - new), np.exp(float(i[t]) - new)
        state, norm, m = a * state + b * torch.outer(k[t], v[t]), a * norm + b * k[t], new
    return rows, state, norm, m


def memory_case(where, heads, dim, vdim, rot, gated, chunks, cap=6.0, spread=2.0, decays=None, seed=0):
    device, dt = where
    r = gen(heads * 100 + dim + seed)
    si, order, _ = step_of(chunks, device)
    t, rows, base = si.num_tokens, H.state_rows(dim), 50.0
    ld = up8(heads * (2 * dim + vdim) + 3)
    full = [r(a + n, ld).to(dt) for a, n in order]
    logits = [spread * r(a + n, 2 * heads + 1) for a, n in order]
    bias = torch.cat([r(heads), 1.5 + r(heads)])
    decay = None if gated else torch.tensor(decays or [1 - 2.0 ** -(1 + 2 * h) for h in range(heads)], dtype=torch.float64)
    q_scale, k_scale = (dim ** -0.5, 1.0) if gated else (1.0, dim ** -0.5)
    state, peak = torch.full((len(order), heads, vdim + gated, rows), 9.0), torch.full((len(order), heads), 9.0)
    state[..., dim:] = 0
    want, left = {}, {}
    for e, slot, _, a, n in entries(si, order):
        x = full[e].double()
        gi = gf = None
        if gated:
            z = cap * torch.tanh((logits[e][:, :2 * heads].double() + bias.double()) / cap)
            gi, gf = z[:, :heads], O.log_sigmoid(z[:, heads:])
        for h in range(heads):
            part = lambda at, w: x[:, at + h * w:at + (h + 1) * w]
            q, k, v = part(0, dim), part(heads * dim, dim), part(2 * heads * dim, vdim)
            q, k = (O.rotate_halves(y, rot, base) for y in (q, k))
            args = lambda m: (q[:m] * q_scale, k[:m] * k_scale, v[:m], gi[:m, h] if gated else None, gf[:m, h] if gated else None, None if gated else float(decay[h]))
            if a > 0:
                _, s0, n0, m0 = memory_after(*args(a))
                state[slot, h, :vdim, :dim] = s0.T.float()
                if gated:
                    state[slot, h, vdim, :dim], peak[slot, h] = n0.float(), m0
            res = memory_after(*args(a + n))
            want[e, h], left[e, h] = res[0][a:], res[1:]
    row = torch.cat([full[e][a:] for e, (a, n) in enumerate(order)]).to(device)
    lg = torch.cat([logits[e][a:] for e, (a, n) in enumerate(order)]).to(device) if gated else None
    turns = None
    if rot:
        turns = H.turn_table(si.positions, hybrid.rotation(rot, base, device), torch.zeros(t, rot // 2, 2, device=device))
    pack = hybrid.pack_memory(hybrid.MemorySpec(heads, dim, vdim, decay=tuple(decay.tolist())), *(torch.zeros(8, 8),) * 5).decay if not gated else None
    state, peak, out = state.to(device), peak.to(device), torch.zeros(t, heads * vdim, device=device)
    H.decay_memory(row, turns, lg, bias.to(device) if gated else None, cap, None if gated else pack.to(device), state, peak if gated else None, out, heads, dim, vdim,
                   q_scale, k_scale, si, blocks=dt == torch.bfloat16)
    if device == "cuda":
        ops.check_status()
    for e, slot, b, a, n in entries(si, order):
        for h in range(heads):
            w = want[e, h]
            err = (out[b:b + n, h * vdim:(h + 1) * vdim].cpu().double() - w).abs().amax(1) / w.abs().amax(1).clamp(min=1e-3 * float(w.abs().max()))
            assert err.max() < 3e-4 and err.median() < 3e-5, (e, h, float(err.max()), int(err.argmax()))
            s, norm, m = left[e, h]
            got = state[slot, h].cpu().double()
            assert (got[:vdim, :dim].T - s).abs().max() < 2e-5 * max(1.0, float(s.abs().max())), (e, h)
            if gated:
                assert (got[vdim, :dim] - norm).abs().max() < 2e-5 * max(1.0, float(norm.abs().max())) and abs(float(peak[slot, h]) - m) < 1e-4, (e, h)
    assert not state[..., dim:].any()


MEMORY_SIZES = [(2, 64, 64, 32), (3, 20, 28, 12), (2, 128, 128, 128), (1, 200, 130, 100), (2, 10, 6, 10), (4, 32, 70, 0), (1, 256, 300, 64), (2, 66, 200, 8)]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("heads,dim,vdim,rot", MEMORY_SIZES)
@pytest.mark.parametrize("gated", [False, True])
def test_memories_along_sequences(where, heads, dim, vdim, rot, gated):
    """Sequences that begin or go on, beside decoded tokens; slots hold anything before a sequence begins."""
    memory_case(where, heads, dim, vdim, 0 if gated else rot, gated, CHUNKS)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("chunks", [[(63, 1)], [(64, 1)], [(0, 63)], [(0, 64)], [(0, 65)], [(1, 64)], [(64, 2)], [(0, 600), (300, 1), (10, 129)]])
@pytest.mark.parametrize("gated", [False, True])
def test_memories_at_block_edges(where, chunks, gated):
    memory_case(where, 2, 32, 40, 0 if gated else 16, gated, chunks)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("decays", [[1.0, 0.0], [0.5, 1e-6], [0.9999, 1 - 2.0 ** -20]])
def test_decays_that_keep_or_forget_everything(where, decays):
    memory_case(where, 2, 24, 16, 8, False, [(0, 300), (70, 1), (5, 66)], decays=decays)


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("cap,spread", [(1.0, 5.0), (15.0, 12.0), (40.0, 40.0)])
def test_gates_far_from_zero(where, cap, spread):
    """Gates at their caps, memories that forget in one token or hardly at all: no exponential overflows, the running maximum counts."""
    memory_case(where, 2, 24, 16, 0, True, [(0, 200), (70, 1), (5, 66)], cap=cap, spread=spread)


@pytest.mark.parametrize("where", WHERE[:2])
def test_rotations_at_far_positions(where):
    device, _ = where
    pos = torch.tensor([0, 1, 17, 4095, 100003, 1048575], dtype=torch.int32)
    got = H.turn_table(pos.to(device), hybrid.rotation(24, 1e6, device), torch.zeros(6, 12, 2, device=device)).cpu()
    unit = torch.zeros(1, 24, dtype=torch.float64)
    unit[0, :12] = 1
    for i, p in enumerate(pos.tolist()):
        want = O.rotate_halves(unit, 24, 1e6, p)[0]
        assert (got[i, :, 0].double() - want[:12]).abs().max() < 2e-7 and (got[i, :, 1].double() - want[12:]).abs().max() < 2e-7


# ------------------------------------------------------------------------------------------
# whole models
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", ENGINES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_layers(models, name, where):
    cfg, tensors = model_for(models, name, where)
    ids = tokens_of(cfg, 150, 1)
    layers = []
    want = O.forward(cfg, tensors, ids, layers_out=layers)
    eng = make_engine(cfg, tensors, where)
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


@GPU
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_long_prompts_in_two_kernel_passes(models, dtype):
    """More rows a step than one pass of norm and convolution takes, in one portion and in several."""
    where = ("cuda", dtype)
    cfg, tensors = model_for(models, "wide", where)
    ids = tokens_of(cfg, 700, 12)
    want = O.forward(cfg, tensors, ids)
    for cuts in ([700], [600, 1, 3, 96]):
        assert_logits(replay_cuts(make_engine(cfg, tensors, where, max_tokens=704), ids, cuts), want, where)


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


@pytest.mark.parametrize("where", ENGINES[:2])
@pytest.mark.parametrize("at", [0, 1, 2, 15, 16, 63, 64, 100, 176, 178])
def test_single_tokens_show_in_logits(models, where, at):
    """Prompts that differ in one token -- the first ones, at page borders, far away, and just inside the input convolutions -- under
    sharpened attention; the oracle itself tells them apart by far more than the tolerance."""
    cfg, tensors = models["wide"]
    tensors = {k: v * 2 if k.endswith("q.norm") else v for k, v in tensors.items()}
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
    """Mistakes planted in the oracle -- filters one tap off, gates, biases, sinks, norms or corrections left out, other constants, a window
    one token off, neighbours rotated instead of halves, a maximum that starts at minus infinity -- move the logits by more than any tolerance."""
    cfg, tensors = models["mixed"]
    ids = tokens_of(cfg, 60, 3)
    want = O.forward(cfg, tensors, ids)
    spread = lambda got: float((got - want).pow(2).mean(-1).sqrt().max() / want.std())
    broken = {"taps": {k: v.roll(1, 1) if "canon" in k else v for k, v in tensors.items()}}
    for end in (".g", ".sink", ".q.b", ".k.b", ".o.b", ".rg1", ".rg1.b", ".rg2", ".rg2.b", ".correction", "mix.i", "mix.i.b", "mix.f", "mix.f.b"):
        broken[end] = {k: v * 0 if k.endswith(end) else v for k, v in tensors.items()}
    for end in ("q.norm", "k.norm", "mix.norm", "norm1", "final.norm"):
        broken[end] = {k: v * 0 + 1 if k.endswith(end) else v for k, v in tensors.items()}
    for what, t in broken.items():
        assert spread(O.forward(cfg, t, ids)) > 5e-3, what

    def other(*path, value):
        c = json.loads(json.dumps(cfg))
        at = c
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        return spread(O.forward(c, tensors, ids))

    assert other("norm", "groups", value=2) > 5e-3 and other("norm", "eps", value=0.1) > 1e-3 and other("embedding", "scale", value=1.0) > 5e-3
    for i, path, value in ((0, ("mask", "size"), 20), (0, ("mask", "size"), 22), (0, ("softcap",), 30.0), (0, ("scale",), 0.1), (1, ("rot", "dims"), 20), (1, ("rot", "base"), 3.0),
                           (1, ("decay",), [0.5, 0.9, 0.99]), (3, ("gate_cap",), 12.0)):
        assert other("layers", i, "mixer", *path, value=value) > 1e-3, path
    assert other("layers", 3, "mlp", "router", "groups", "keep", value=2) > 1e-3 and other("layers", 3, "mlp", "router", "top", value=2) > 1e-3

    def planted(name, fn):
        with monkeypatch.context() as m:
            m.setattr(O, name, fn)
            return spread(O.forward(cfg, tensors, ids))

    plain = O.rotate_halves
    assert planted("rotate_halves", lambda x, dims, base, start=0: torch.cat([plain(x[:, :dims].reshape(len(x), -1, 2).transpose(1, 2).reshape(len(x), -1), dims, base, start), x[:, dims:]], 1)) > 5e-3
    assert planted("slope", lambda a, heads: 2.0 ** (-8.0 * a / heads)) > 5e-3
    head = O.matrix_memory_head
    assert planted("matrix_memory_head", lambda q, k, v, i, f: head(q, k, v, i + 3, f)) > 1e-3
    attend = O.attention_head
    assert planted("attention_head", lambda q, k, v, *a: attend(q, k, k, *a)) > 5e-3              # values that went through the norm
    assert planted("sublayer_input", lambda h, w: O.causal_filter(h, w)) > 5e-3


# ------------------------------------------------------------------------------------------
# serving: directory, scheduler, generation
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_in_batches(models, device, graphs, tmp_path):
    if graphs and device == "cpu":
        pytest.skip("CUDA graphs")
    cfg, tensors = models["mixed"]
    d = write_checkpoint(tmp_path / "m", cfg, tensors)
    eng = Engine.from_dir(d, device=device, max_seqs=3, max_seq_len=300, num_pages=60, max_tokens_per_step=64, compute_dtype="f32", cuda_graphs=graphs)
    prompts = [tokens_of(cfg, n, 50 + n) for n in (5, 90, 1, 40, 17)]
    res = eng.generate_batch(prompts, GenerateOptions(max_new_tokens=24, greedy=True, ignore_eos=True))
    for p, r in zip(prompts, res):
        assert len(r.token_ids) == 24 and O.follows_greedily(cfg, tensors, p, r.token_ids)
    if graphs:
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
    cfg, tensors = models["mixed"]
    eng = make_engine(cfg, tensors, (device, "f32"), max_tokens=224, max_seqs=4, num_pages=10, max_tokens_per_step=64, prefill_chunk=64, max_logit_rows=0)
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
    read = registry.ARCHITECTURES["Midisun"].read_config
    cfg = read(MIXED)
    w = registry.family_of(cfg).random_weights(cfg, "cpu", 1, 0, 0, torch.float32)
    assert w.embed_norm is None and w.layers[0].gate1 is not None and w.layers[2].gate2 is None and w.layers[0].conv2 is None and w.layers[3].moe.bias is not None
    assert w.layers[1].mixer.decay.shape == (2, 3) and w.layers[2].mixer.gates.shape[0] == 4
    eng = replay.Replayer(checkpoint_helpers.LLMEngine(checkpoint_helpers.EngineConfig(model=cfg, num_pages=16, max_seqs=2, max_seq_len=64, compute_dtype="f32"), weights=w, device="cpu"))
    assert torch.isfinite(eng.step([{"id": "a", "tokens": [1, 2, 3], "want": [2]}], ["a"])[0]).all()
    assert cfg.sliding_window == 50 and cfg.attention_sinks == 0 and cfg.kv_bytes_per_token() == 2 * (2 * 24 + 2 + 4 * 16 + 2) and cfg.weight_bytes() > 0
    assert [sorted(cfg.state_shapes(i)) for i in range(3)] == [["input1"], ["input1", "recurrent"], ["input1", "peak", "recurrent"]]


def test_configurations_that_cannot_run_are_refused(models):
    cfg, tensors = models["mixed"]
    read = registry.ARCHITECTURES["Midisun"].read_config
    for path, value, what in ((("layers", 0, "type"), "other", "mixer type"), (("canon", "taps"), 9, "taps"), (("layers", 1, "mixer", "rot", "dims"), 22, "rotated"),
                              (("layers", 0, "mlp", "kind"), "other", "feed-forward"), (("layers", 1, "mlp", "router", "top"), 5, "cannot be chosen"),
                              (("norm", "groups"), 5, "groups"), (("layers", 1, "mixer", "decay"), [0.5], "decays"), (("layers", 1, "mixer", "decay"), [0.5, 0.5, 1.5], "decays"),
                              (("layers", 0, "mixer", "vdim"), 10, "values"), (("layers", 0, "mixer", "kv_heads"), 4, "divide"), (("layers", 2, "mixer", "dim"), 300, "recurrent key width"),
                              (("layers", 1, "mlp", "router", "groups", "count"), 4, "equal groups")):
        bad = json.loads(json.dumps(cfg))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError, match=what):
            read(bad)
    c, load = read(cfg), registry.ARCHITECTURES["Midisun"].load_weights
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
    assert json.loads(capsys.readouterr().out)["architecture"]["name"] == "Midisun"
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
