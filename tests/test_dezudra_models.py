"""Dezudra decoders (differential attention, gated delta rule, short convolutions, squared-relu experts): every mechanism, the whole
model and the serving path against the plain statement in oracle_dezudra.py, on the CPU path and -- marked gpu -- on the
kernels, in 32-bit and in bf16."""
import io
import json

import checkpoint_helpers
import numpy as np
import oracle_dezudra as O
import pytest
import torch
from checkpoint_helpers import CHUNKS, DEVICES, ENGINES, GPU, make_engine, replay_cuts, step_of, tokens_of, write_checkpoint

from onnx_genai_b200 import ops, replay
from onnx_genai_b200.engine.api import Engine, GenerateOptions
from onnx_genai_b200.models import registry
from onnx_genai_b200.ops import hybrid as H
from onnx_genai_b200.ops import moe as M
from onnx_genai_b200.ops import reference

X = O.experts
# sizes that are no multiples of 8, several windows and kept prefixes, layers without a feed-forward, one group and many
MIXED = O.make_config(97, 72, [O.layer_attention(4, 2, 20, 28, 21, 5, X(6, 2, 40, 3, 2), rot=12, base=500.0), O.layer_delta(4, 2, 20, 36, X(5, 1, 24), conv=4),
                               O.layer_attention(3, 1, 16, 24, 50, 19, None, conv=2, diff=0.7, scale=0.4), O.layer_delta(3, 3, 40, 12, None, conv=2),
                               O.layer_attention(2, 2, 12, 10, 9, 0, X(8, 3, 16, 4, 3), conv=5, diff=0.2)], eps=1e-4, logit_scale=0.7)
ODD = O.make_config(61, 50, [O.layer_attention(1, 1, 10, 14, 33, 1, X(3, 3, 35), rot=6, conv=1), O.layer_delta(1, 1, 70, 5, X(4, 2, 9, 2, 1), conv=1),
                             O.layer_attention(5, 1, 6, 18, 17, 30, X(2, 1, 20), rot=2, conv=6)], eps=1e-3, logit_scale=3.0)
RECURRENT = O.make_config(64, 64, [O.layer_delta(4, 1, 16, 16, X(4, 2, 64, 2, 2)), O.layer_delta(2, 2, 130, 40, X(4, 2, 64, 4, 2), conv=3),
                                   O.layer_delta(4, 4, 64, 128, None)])
# shapes of the tensor-core kernels
WIDE = O.make_config(80, 128, [O.layer_attention(8, 2, 64, 128, 70, 33, X(8, 2, 128, 4, 2)), O.layer_attention(16, 1, 32, 64, 128, 0, X(4, 1, 64)),
                               O.layer_delta(4, 2, 128, 128, X(8, 4, 64, 2, 2)), O.layer_attention(2, 2, 128, 128, 200, 16, None, rot=64),
                               O.layer_attention(3, 1, 96, 192, 45, 7, None)])
# heads in steps of the vector width beside key widths and channel counts that are not
UNEVEN = O.make_config(70, 68, [O.layer_delta(3, 3, 7, 128, X(4, 2, 20, 2, 1), conv=3), O.layer_attention(2, 1, 9, 64, 30, 6, X(3, 1, 12), rot=4, conv=4),
                                O.layer_delta(2, 1, 64, 9, None, conv=5), O.layer_attention(9, 3, 64, 20, 18, 2, None, rot=22)])
CONFIGS = {"mixed": MIXED, "odd": ODD, "recurrent": RECURRENT, "wide": WIDE, "uneven": UNEVEN}
WHERE = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=GPU), pytest.param(("cuda", torch.bfloat16), marks=GPU)]


@pytest.fixture(scope="module")
def models():
    return {name: (cfg, O.random_tensors(cfg, seed=20 + i)) for i, (name, cfg) in enumerate(CONFIGS.items())}


def assert_logits(got, want, where):
    checkpoint_helpers.assert_logits(got, want, where, outliers=0.02)


def model_for(models, name, where):
    """In bf16 every expert is used, since rounding could tip a close choice (choosing is tested on fixed logits), and attention is
    less sharp, which magnifies rounding less."""
    cfg, tensors = models[name]
    if where[1] == "bf16":
        cfg, tensors = json.loads(json.dumps(cfg)), O.random_tensors(cfg, seed=40, sharp=1.0)
        for layer in cfg["layers"]:
            if layer["mlp"]:
                r = layer["mlp"]["router"]
                r["top"], r["groups"]["keep"] = r["experts"], r["groups"]["count"]
    return cfg, tensors


def entries(si, order):
    """(sequence index, slot, first row, tokens before, rows) of a hand-made plan."""
    base, slots = 0, si.state_slot.cpu()
    for e, (a, n) in enumerate(order):
        yield e, int(slots[e]), base, a, n
        base += n


# ------------------------------------------------------------------------------------------
# mechanisms
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("width,k", [(40, 0), (37, 3), (1100, 2), (4096, 0), (20, 1), (2050, 5)])
def test_norm_step(device, width, k):
    """x + post(y), then the norm; y a row, or a weighted sum of expert rows."""
    g = torch.Generator().manual_seed(width)
    r = lambda *s: torch.randn(*s, generator=g)
    t, eps, ld = 9, 1e-3, width + (-width) % 8
    x, post, w = r(t, width), H.RmsNorm(r(width), eps), H.RmsNorm(r(width), eps)
    if k:
        rows, pos = r(t * k + 4, ld), torch.randperm(t * k + 4, generator=g)[:t * k].int().view(t, k)
        weight = torch.rand(t, k, generator=g)
        y = (rows[pos.long()] * weight[:, :, None]).sum(1)[:, :width]
        src = H.ExpertRows(rows.to(device), pos.to(device), weight.to(device))
    else:
        full = r(t, ld)
        y, src = full[:, :width], full.to(device)
    d = lambda n: H.RmsNorm(n.w.to(device), n.eps)
    xd, h = x.clone().to(device), torch.zeros(t, ld, device=device)
    pick = torch.tensor([8, 0, 5], dtype=torch.int32)
    hl = torch.zeros(3, ld, device=device)
    H.norm_step(xd, src, d(post), d(w), hl, gather=pick.to(device))
    assert torch.equal(xd.cpu(), x)                       # rows picked for the output leave the residual alone
    H.norm_step(xd, src, d(post), d(w), h)
    want = (x + O.rms_norm(y, post.w, eps)).double()
    torch.testing.assert_close(xd.cpu().double(), want, atol=2e-5, rtol=1e-5)
    torch.testing.assert_close(h.cpu().double()[:, :width], O.rms_norm(want, w.w.double(), eps), atol=4e-5, rtol=2e-5)
    torch.testing.assert_close(hl.cpu(), h.cpu()[pick.long()], atol=1e-6, rtol=1e-6)


def conv_case(g, order, channels, taps):
    """Inputs, filter, what came before every sequence, and the convolved rows: (u, w, history, y, last inputs)."""
    w = torch.randn(channels, taps, generator=g)
    u, past, y, last = [], [], [], []
    for a, n in order:
        seq = torch.randn(a + n, channels, generator=g)
        y.append(O.causal_conv(seq, w)[a:])
        pad = torch.cat([torch.zeros(taps, channels), seq])
        past.append(pad[a + taps - (taps - 1):a + taps] if taps > 1 else pad[:0])
        last.append(pad[a + n + taps - (taps - 1):] if taps > 1 else pad[:0])
        u.append(seq[a:])
    return torch.cat(u), w, past, y, last


SIZES = [(2, 1, 1, 24, 16, 12), (6, 2, 1, 20, 28, 20), (4, 4, 2, 10, 6, 6), (2, 2, 3, 64, 128, 64), (1, 1, 1, 8, 4, 0)]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("nq,nk,nv,d,dv,rot", SIZES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 8])
def test_conv_rope_append(where, nq, nk, nv, d, dv, rot, taps):
    device, dt = where
    g = torch.Generator().manual_seed(taps + d)
    si, order, pages = step_of(CHUNKS, device)
    t, C = si.num_tokens, (nq + nk) * d + nv * dv
    dp, vp, base = d + (-d) % 8, dv + (-dv) % 8, 300.0
    u, w, past, ys, last = conv_case(g, order, C, taps)
    bias = torch.randn(C, generator=g)
    if dt == torch.bfloat16:                              # rounding that the oracle sees as well
        bias = bias.bfloat16().float()
    ld = C + (-C) % 8
    raw = torch.zeros(t, ld, dtype=dt)
    raw[:, :C] = u - bias
    state = torch.full((len(order), taps - 1, C), 9.0)    # stale: sequences that begin start from zeros
    for e, slot, _, a, _ in entries(si, order):
        if a > 0:
            state[slot] = past[e]
    state = state.to(device)
    q, pool = torch.zeros(t, nq * dp, dtype=dt, device=device), torch.zeros(pages, 16 * (nk * dp + nv * vp), dtype=dt, device=device)
    freq = base ** (-2 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))
    H.conv_rope_append(raw.to(device), w.t().contiguous().to(device), bias.to(device), state, q, pool, freq.to(device), si, nq, nk, nv, d, dv, dp, vp)
    keys, values = reference.diff_pages(pool.cpu(), nk, nv, dp, vp)
    table, tol = si.page_table.cpu().long(), dict(atol=2e-5, rtol=1e-5) if dt == torch.float32 else dict(atol=0.05, rtol=0.02)
    for e, slot, b, a, n in entries(si, order):
        y = ys[e]
        at = torch.arange(a, a + n)
        turn = lambda x: O.rotate(torch.cat([torch.zeros(a, x.shape[1]), x]).double(), rot, base)[a:].float() if rot else x
        for hd in range(nq + nk):
            want = turn(y[:, hd * d:(hd + 1) * d])
            got = q[b:b + n, hd * dp:hd * dp + d].cpu() if hd < nq else keys[table[e, at // 16], hd - nq, at % 16, :d]
            torch.testing.assert_close(got.float(), want, **tol)
        for hd in range(nv):
            c = (nq + nk) * d + hd * dv
            torch.testing.assert_close(values[table[e, at // 16], hd, at % 16, :dv].float(), y[:, c:c + dv], **tol)
        if taps > 1:
            torch.testing.assert_close(state[slot].cpu(), last[e], atol=2e-5 if dt == torch.float32 else 0.03, rtol=1e-2 if dt == torch.bfloat16 else 1e-5)
    assert not keys[..., d:].any() and not values[..., dv:].any()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("nk,nv,d,dv", [(1, 2, 24, 40), (3, 3, 10, 7), (2, 4, 64, 128), (1, 1, 200, 300), (2, 2, 130, 20)])
@pytest.mark.parametrize("taps", [1, 3, 4, 7])
def test_conv_unit_gates(where, nk, nv, d, dv, taps):
    device, dt = where
    g = torch.Generator().manual_seed(taps + d)
    si, order, _ = step_of(CHUNKS, device)
    t, C = si.num_tokens, 2 * nk * d + nv * dv
    u, w, past, ys, last = conv_case(g, order, C, taps)
    u[5] = 0 if taps == 1 else u[5]                       # a head of length zero stays zero
    ld = C + (-C) % 8
    raw = torch.zeros(t, ld, dtype=dt)
    raw[:, :C] = u
    if dt == torch.bfloat16:
        u = raw[:, :C].float()
    state = torch.full((len(order), taps - 1, C), 9.0)
    for e, slot, _, a, _ in entries(si, order):
        if a > 0:
            state[slot] = past[e]
    state = state.to(device)
    ab, a_log, dt_bias = torch.randn(t, 2 * nv + 3, generator=g) * 4, torch.rand(nv, generator=g) * 3 - 2, torch.randn(nv, generator=g)
    ab[2, 0] = 40.0                                       # softplus is the identity up there
    qk, v, gates = torch.zeros(t, 2 * nk * d, device=device), torch.zeros(t, nv * dv, dtype=dt, device=device), torch.zeros(t, nv, 2, device=device)
    H.conv_unit_gates(raw.to(device), w.t().contiguous().to(device), state, ab.to(device), a_log.to(device), dt_bias.to(device), qk, v, gates, si, nk, nv, d, dv)
    tol = dict(atol=1e-5, rtol=1e-4) if dt == torch.float32 else dict(atol=0.02, rtol=0.02)
    for e, slot, b, a, n in entries(si, order):
        seq = torch.cat([past[e], u[b:b + n]])
        y = O.silu(O.causal_conv(seq, w)[taps - 1:])
        x = O.unit(y[:, :2 * nk * d].reshape(n, 2, nk, d))
        torch.testing.assert_close(qk[b:b + n].cpu(), torch.cat([x[:, 0].reshape(n, -1) * d ** -0.5, x[:, 1].reshape(n, -1)], 1), **tol)
        torch.testing.assert_close(v[b:b + n].float().cpu(), y[:, 2 * nk * d:], **tol)
        if taps > 1:
            torch.testing.assert_close(state[slot].cpu(), seq[-(taps - 1):], atol=1e-6, rtol=1e-6)
    torch.testing.assert_close(gates[:, :, 0].cpu(), O.log_decay(ab[:, :nv] + dt_bias, a_log), atol=1e-6, rtol=1e-5)
    torch.testing.assert_close(gates[:, :, 1].cpu(), torch.sigmoid(ab[:, nv:2 * nv]), atol=1e-6, rtol=1e-5)


LONG = [(7, 1), (0, 1), (30, 2), (0, 2), (0, 16), (5, 17), (64, 64), (1, 130), (0, 75), (0, 129), (3, 31), (100, 200)]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("heads,groups,dim,vdim", [(2, 1, 44, 56), (3, 3, 20, 36), (1, 1, 64, 10), (4, 2, 128, 130), (1, 1, 200, 33), (4, 1, 100, 32), (2, 2, 256, 140),
                                                   (2, 2, 128, 128), (6, 2, 64, 64)])
@pytest.mark.parametrize("kind", ["plain", "fast", "closed"])
@pytest.mark.parametrize("blocks", [False, True])
def test_delta_rule(where, heads, groups, dim, vdim, kind, blocks):
    """``fast``: decays near zero; ``closed``: no decay and full steps, keys that repeat (every write replaces one).  ``blocks``:
    prompts in blocks on the tensor cores, as exact as the steps."""
    device, dt = where
    if device == "cpu" and blocks:
        pytest.skip("a variant of the CUDA kernel")
    g = torch.Generator().manual_seed(dim)
    si, order, _ = step_of(LONG, device)
    t = si.num_tokens
    qk = O.unit(torch.randn(t, 2, groups, dim, generator=g))
    v = torch.randn(t, heads * vdim, generator=g).to(dt)
    gates = torch.stack([-torch.rand(t, heads, generator=g) * 0.3, torch.rand(t, heads, generator=g)], -1)
    if kind == "fast":
        gates[..., 0] *= 100
        gates[3::7, :, 0] = -200.0                        # the decay underflows to zero: the state starts over
    if kind == "closed":
        gates[..., 0], gates[..., 1] = 0, 1
        qk[:, 1] = qk[torch.randint(0, 6, (t,), generator=g), 1]
    qk[:, 0] *= dim ** -0.5
    rows = H.state_rows(dim)
    start = torch.randn(len(order), heads, vdim, rows, generator=g)
    start[..., dim:] = 0
    state, out = start.to(device).clone(), torch.zeros(t, heads * vdim, device=device)
    H.delta_rule(qk.reshape(t, -1).to(device), v.to(device), gates.to(device), state, out, heads, groups, dim, vdim, si, blocks=blocks)
    for e, slot, b, a, n in entries(si, order):
        for h in range(heads):
            q, k = (qk[b:b + n, i, h // (heads // groups)].double() for i in range(2))
            x = v[b:b + n, h * vdim:(h + 1) * vdim].double()
            S = start[slot, h, :, :dim].double().T if a > 0 else torch.zeros(dim, vdim, dtype=torch.float64)
            want = []
            for i in range(n):
                S = torch.exp(gates[b + i, h, 0].double()) * S
                S = S + torch.outer(k[i], gates[b + i, h, 1].double() * (x[i] - S.T @ k[i]))
                want.append(S.T @ q[i])
            want = torch.stack(want)
            err = (out[b:b + n, h * vdim:(h + 1) * vdim].cpu().double() - want).abs().max() / want.abs().max()
            assert err < 5e-5, (e, h, float(err))
            assert (state[slot, h, :, :dim].cpu().double().T - S).abs().max() < 5e-5 * max(1.0, float(S.abs().max())), (e, h)
    assert not state[..., dim:].any()


def diff_case(where, hq, hkv, d, dv, window, keep, chunks, spike, splits=1, counters=None):
    """Differential attention over random pages; ``spike``: one key of each map outshines the others at a position."""
    device, dt = where
    g = torch.Generator().manual_seed(hq * 1000 + d)
    si, order, pages = step_of(chunks, device, page_seed=3)
    dp, vp = d + (-d) % 8, dv + (-dv) % 8
    pool = torch.zeros(pages, 16 * hkv * (2 * dp + vp))
    keys, values = reference.diff_pages(pool, 2 * hkv, hkv, dp, vp)
    table, t = si.page_table.cpu().long(), si.num_tokens
    q, kv = torch.randn(t, hq, 2, d, generator=g), []
    if spike is not None:
        q = 0.7 + 0.05 * q
    for e, (a, n) in enumerate(order):
        k, v = torch.randn(a + n, hkv, 2, d, generator=g) * 0.5, torch.randn(a + n, hkv, dv, generator=g)
        if spike is not None:
            for m in range(2):                            # the two maps look at different keys
                at = spike(a + n) - m
                if 0 <= at < a + n:
                    k[at, :, m] = 12.0 / d ** 0.5
        k, v = k.to(dt).float(), v.to(dt).float()
        j = torch.arange(a + n)
        keys[table[e, j // 16], :, j % 16, :d] = k.reshape(a + n, 2 * hkv, d)
        values[table[e, j // 16], :, j % 16, :dv] = v
        kv.append((k.double(), v.double()))
    if window > 0:                                        # pages that no query sees are gone
        for e, (a, n) in enumerate(order):
            si.page_table[e, -(-keep // 16):max(-(-keep // 16), (a - window + 1) // 16)] = -1
    q = q.to(dt)
    qp = torch.zeros(t, hq, 2, dp, dtype=dt)
    qp[..., :d] = q
    out = torch.zeros(t, hq * vp, dtype=dt, device=device)
    part_o, part_ml = torch.empty(t * hq * 32 * splits * vp, device=device), torch.empty(t * hq * 64 * splits, device=device)
    scale, lam, eps, gain = 1.3 * d ** -0.5, 0.6, 1e-4, 0.45
    H.diff_attention(qp.view(t, -1).to(device), out, pool.to(dt).to(device), si, hq, hkv, d, dv, dp, vp, scale, lam, eps, gain, window, keep, splits,
                     part_o, part_ml, counters)
    if device == "cuda":
        ops.check_status()
    for e, slot, b, a, n in entries(si, order):
        k, v = kv[e]
        seen = O.visible(a + n, window, keep)[a:]
        for h in range(hq):
            c = h // (hq // hkv)
            maps = [O.softmax_attention(q[b:b + n, h, m].double(), k[:, c, m], v[:, c], scale, seen) for m in range(2)]
            want = O.rms_norm(maps[0] - lam * maps[1], None, eps) * gain
            got = out[b:b + n, h * vp:h * vp + dv].cpu().double()
            assert (got - want).abs().max() < (0.03 if dt == torch.bfloat16 else 3e-5), (e, h, int((got - want).abs().amax(1).argmax()))


DIFF_SIZES = [(3, 1, 20, 28, 21, 5), (1, 1, 10, 6, 1, 0), (4, 2, 64, 128, 70, 33), (8, 1, 32, 64, 100, 16), (20, 1, 48, 96, 64, 1), (2, 2, 128, 128, 130, 0),
              (2, 1, 96, 192, 40, 50), (2, 2, 16, 256, 30, 7), (6, 3, 64, 64, 0, 0), (1, 1, 130, 300, 33, 20)]


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("hq,hkv,d,dv,window,keep", DIFF_SIZES)
def test_diff_attention_edges(where, hq, hkv, d, dv, window, keep):
    """Random keys, and keys that stand out just inside and just outside the window and the kept prefix, at the first
    token, at page borders and far away."""
    chunks = [(7, 1), (0, 1), (window + 40, 1), (300, 1), (30, 2), (0, 2), (5, 17), (210, 70), (0, 150), (250, 3)]
    diff_case(where, hq, hkv, d, dv, window, keep, chunks, None)
    spots = [lambda n: 1, lambda n: 16, lambda n: n - 1]
    if window > 0:
        spots += [lambda n: n - window, lambda n: n - 1 - window, lambda n: n - window + 1, lambda n: keep - 1, lambda n: keep, lambda n: keep + 1]
    for spot in spots:
        diff_case(where, hq, hkv, d, dv, window, keep, chunks, spot)


@GPU
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hq,hkv,d,dv,window,keep,splits", [(3, 1, 24, 28, 0, 0, 4), (8, 2, 64, 128, 300, 40, 3), (4, 4, 128, 128, 200, 0, 8), (18, 1, 64, 64, 0, 0, 5)])
def test_diff_decode_with_split_keys(dtype, hq, hkv, d, dv, window, keep, splits):
    chunks = [(7, 1), (0, 1), (400, 1), (255, 1), (15, 1), (16, 1), (299, 1), (300, 1), (900, 1)]
    counters = torch.zeros(len(chunks) * hq, dtype=torch.int32, device="cuda")
    for spot in (None, (lambda n: n - window) if window else (lambda n: 20), lambda n: 1, lambda n: keep - 1):
        for _ in range(2):                                # the counters come back as zeros
            diff_case(("cuda", dtype), hq, hkv, d, dv, window, keep, chunks, spot, splits, counters)
    assert (counters == 0).all()


@pytest.mark.parametrize("where", WHERE)
@pytest.mark.parametrize("experts,top,groups,keep,hidden,inter,tokens", [(6, 2, 3, 2, 40, 24, 9), (8, 4, 4, 3, 72, 40, 150), (5, 1, 1, 1, 20, 8, 3), (64, 6, 8, 3, 128, 64, 300),
                                                                         (4, 4, 2, 2, 264, 136, 1), (256, 8, 16, 1, 64, 72, 40)])
def test_squared_relu_experts_in_groups(where, experts, top, groups, keep, hidden, inter, tokens):
    from onnx_genai_b200.models.hybrid import pack_moe

    device, dt = where
    g = torch.Generator().manual_seed(experts)
    h = torch.randn(tokens, hidden, generator=g).to(dt)
    W = {"router": torch.randn(experts, hidden, generator=g) * 2 / hidden ** 0.5}
    for e in range(experts):
        W[f"e{e}.up"], W[f"e{e}.down"] = (torch.randn(inter, hidden, generator=g) / hidden ** 0.5).to(dt), (torch.randn(hidden, inter, generator=g) / inter ** 0.5).to(dt)
    w = pack_moe(W["router"].to(dt), [W[f"e{e}.up"] for e in range(experts)], [W[f"e{e}.down"] for e in range(experts)])
    hp = torch.zeros(tokens, w.up.shape[2], dtype=dt)
    hp[:, :hidden] = h
    logits = (h.double() @ W["router"].double().T).float()
    ws = M.MoEWorkspace(tokens, top, experts, w.up.shape[2], w.up.shape[1], device, dt)
    y = M.relu2_experts(hp.to(device), logits.to(device), w.up.to(device), w.down.to(device), ws, top, groups, keep)
    got = (y.rows[y.pos.long()].float() * y.weight[:, :, None]).sum(1)[:, :hidden].cpu().double()
    cfg = {"router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}
    want = O.experts_forward(h.double(), {k: v.double() for k, v in W.items()}, cfg)
    assert (got - want).abs().max() < (2e-5 if dt == torch.float32 else 0.02) * want.abs().max()


def test_choice_of_groups_matters():
    """A group with two good experts loses to groups with one better each: the oracle and the op agree on who stays."""
    logits = torch.tensor([[3.0, 2.9, 4.0, -9.0, 3.5, -9.0]])
    ids, w = reference.moe_route(logits, 3, False, 3, 2)
    assert sorted(ids[0].tolist()) in ([2, 3, 4], [2, 4, 5]) and O.choose_experts(torch.softmax(logits[0], 0), 2, 3, 2) == [2, 4]
    assert torch.allclose(w[0, :2], torch.softmax(logits[0], 0)[[2, 4]])      # not renormalised
    plain, _ = reference.moe_route(logits, 3, False)
    assert sorted(plain[0].tolist()) == [0, 2, 4]


# ------------------------------------------------------------------------------------------
# the whole model through the engine
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
    assert len(eng.model.capture) == len(cfg["layers"])
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


@pytest.mark.parametrize("where", ENGINES)
def test_window_releases_pages_but_keeps_the_first(models, where):
    """Pages behind the widest window go back to the pool while a sequence runs, except those of the kept first tokens; a long
    sequence needs no more than both."""
    cfg, tensors = model_for(models, "mixed", where)                        # windows 21, 50 and 9, kept 5, 19 and 0: two pages stay
    ids = tokens_of(cfg, 260, 5)
    eng = make_engine(cfg, tensors, where, max_tokens=144, max_seq_len=400)
    sid_pages = []
    rep, rows, at = replay.Replayer(eng), [], 0
    for n in [9, 1, 1, 14, 2, 30, 3] * 5:
        n = min(n, len(ids) - at)
        if n:
            rows += rep.step([{"id": "a", "tokens": ids[at:at + n], "want": list(range(n))}], [])
            at += n
            sid_pages.append(eng.core.released_pages(rep.open["a"]))
    assert at == 260 and sid_pages[-1] > 8
    assert_logits(torch.stack(rows), O.forward(cfg, tensors, ids), where)


@pytest.mark.parametrize("where", ENGINES[:2])
@pytest.mark.parametrize("gap", ["window", "kept", "far"])
def test_single_far_keys_show_in_logits(models, where, gap):
    """Prompts that differ in one token just inside or outside the window of the last one, just inside or outside the kept
    prefix, or far behind both, under sharpened attention."""
    cfg, tensors = models["wide"]
    tensors = dict(tensors)
    for i in (0, 1, 3, 4):
        tensors[f"l{i}.mix.q"] = tensors[f"l{i}.mix.q"] * 2
    m = cfg["layers"][0]["mixer"]["mask"]
    base = tokens_of(cfg, 180, 6)
    spots = {"window": (180 - m["size"], 179 - m["size"]), "kept": (m["keep_first"] - 1, m["keep_first"]), "far": (0, 60)}[gap]
    for at in spots:
        for tok in (3, 4):
            ids = list(base)
            ids[at] = tok
            assert_logits(replay_cuts(make_engine(cfg, tensors, where), ids, [50, 2, 60, 66, 1]), O.forward(cfg, tensors, ids), where)


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
    r = eng.generate(prompts[0], GenerateOptions(max_new_tokens=150, greedy=True, ignore_eos=True))      # long decoding, far past every window
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
    cfg, tensors = models["wide"]
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


def test_configurations_that_cannot_run_are_refused(models):
    cfg, tensors = models["odd"]
    read = registry.ARCHITECTURES["Dezudra"].read_config
    for path, value, what in ((("layers", 0, "type"), "other", "mixer type"), (("layers", 0, "mixer", "conv"), 9, "taps"), (("layers", 0, "mixer", "rot", "dims"), 5, "rotated"),
                              (("layers", 2, "mixer", "kv_heads"), 2, "key heads"), (("layers", 0, "mlp", "kind"), "dense", "feed-forward"),
                              (("layers", 1, "mlp", "router", "top"), 3, "cannot be chosen"), (("layers", 1, "mlp", "router", "groups", "count"), 3, "groups")):
        bad = json.loads(json.dumps(cfg))
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError, match=what):
            read(bad)
    c, load = read(cfg), registry.ARCHITECTURES["Dezudra"].load_weights
    assert load(c, {**tensors, "l9.extra": torch.zeros(1)}, torch.float32, "cpu").unused == ["l9.extra"]
    with pytest.raises(KeyError, match="l0.norm1b"):
        load(c, {k: v for k, v in tensors.items() if k != "l0.norm1b"}, torch.float32, "cpu")
    for kw, what in (({"max_draft_tokens": 2}, "speculative"), ({"kv_dtype": "fp8"}, "fp8")):
        with pytest.raises(ValueError, match=what):
            make_engine(cfg, tensors, ("cpu", "f32"), **{"compute_dtype": "bf16", **kw})


def test_directory_commands_and_replay(models, tmp_path, capsys):
    from onnx_genai_b200 import cli

    cfg, tensors = models["odd"]
    d = write_checkpoint(tmp_path / "m", cfg, tensors)
    assert cli.main(["show", d]) == 0
    assert json.loads(capsys.readouterr().out)["architecture"]["name"] == "Dezudra"
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
