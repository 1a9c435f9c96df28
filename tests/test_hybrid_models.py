"""Models with a mixer per layer (Rilelorn): every mechanism, the whole model and the serving path against the plain
statement in oracle_rilelorn.py, on the CPU path and -- marked gpu -- on the kernels, in 32-bit and in bf16."""
import io
import json

import numpy as np
import oracle_rilelorn as O
import pytest
import torch
from checkpoint_helpers import CHUNKS, DEVICES, ENGINES, GPU, assert_logits, make_engine, replay_cuts, step_of, tokens_of, write_checkpoint

from onnx_genai_b200 import ops, replay
from onnx_genai_b200.engine.api import Engine, GenerateOptions
from onnx_genai_b200.engine.core import Core, CoreConfig
from onnx_genai_b200.models import registry
from onnx_genai_b200.ops import hybrid as H
from onnx_genai_b200.package.safetensors import SafetensorsFile

# sizes that are no multiples of 8, more than one window, a shared cache read with other heads, layers without a feed-forward
MIXED = O.make_config(97, 72, 3, [O.layer_latent(3, 24, 40, 56, 21, 80), O.layer_hgrn2(3, 20, 36, 96),
                                  O.layer_latent(5, 16, 24, 56, 9, 0, scale=0.31, kv_from=0), O.layer_hgrn2(2, 40, 12, 0),
                                  O.layer_latent(2, 12, 10, 20, 50, 36)], eps=1e-4)
ODD = O.make_config(61, 50, 1, [O.layer_latent(1, 10, 14, 18, 1, 33), O.layer_hgrn2(1, 70, 5, 35), O.layer_latent(2, 10, 6, 18, 17, 20, kv_from=0)])
RECURRENT = O.make_config(64, 64, 2, [O.layer_hgrn2(4, 16, 16, 64), O.layer_hgrn2(2, 130, 40, 64)])
ATTENTION = O.make_config(80, 128, 4, [O.layer_latent(8, 32, 32, 128, 70, 128), O.layer_latent(4, 64, 64, 128, 33, 128, kv_from=0),
                                       O.layer_latent(16, 32, 16, 192, 200, 128)])
# latents wider than a head: prompts run on expanded keys and values in bf16
WIDE = O.make_config(90, 96, 2, [O.layer_latent(3, 64, 64, 136, 37, 64), O.layer_hgrn2(2, 24, 24, 64), O.layer_latent(2, 128, 128, 136, 90, 64, kv_from=0),
                                 O.layer_latent(1, 64, 64, 200, 500, 0)])
CONFIGS = {"mixed": MIXED, "odd": ODD, "recurrent": RECURRENT, "attention": ATTENTION, "wide": WIDE}


@pytest.fixture(scope="module")
def models():
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        out[name] = (cfg, O.random_tensors(cfg, seed=10 + i))
    return out


# ------------------------------------------------------------------------------------------
# mechanisms
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("streams,width", [(1, 40), (2, 64), (3, 37), (4, 1100), (7, 20)])
def test_hyper_step_with_norm_and_shift(device, streams, width):
    g = torch.Generator().manual_seed(streams)
    r = lambda *s: torch.randn(*s, generator=g)
    si, order, _ = step_of(CHUNKS, device)
    t = si.num_tokens
    x, y = r(t, streams, width), r(t, width)
    conn = H.HyperConnection(r(streams), r(streams), r(streams, streams))
    read, norm, amount = r(streams), H.DynamicTanh(torch.tensor([0.7]), r(width), r(width)), torch.rand(width, generator=g)
    prev = r(len(order), width)
    d = lambda v: v.to(device)
    dn = H.DynamicTanh(d(norm.alpha), d(norm.w), d(norm.b))
    dc = H.HyperConnection(d(conn.read), d(conn.write), d(conn.mix))
    x_out, h, state = torch.zeros(t, streams, width, device=device), torch.zeros(t, width, device=device), d(prev.clone())
    H.hyper_step(d(x), x_out, d(y), dc, d(read), dn, h, si, shift=d(amount), prev=state)
    new = O.write_streams(x.permute(1, 0, 2), conn.mix, conn.write, y)
    u = O.dynamic_tanh(O.read_streams(new, read), norm.alpha, norm.w, norm.b)
    torch.testing.assert_close(x_out.cpu(), new.permute(1, 0, 2), atol=2e-5, rtol=1e-5)
    base, slots = 0, si.state_slot.cpu()
    for e, (a, n) in enumerate(order):
        rows = u[base:base + n]
        if a > 0:                       # the row before the chunk comes from the sequence's slot
            want = O.token_shift(torch.cat([prev[slots[e]][None], rows]), amount)[1:]
        else:
            want = O.token_shift(rows, amount)
        torch.testing.assert_close(h[base:base + n].cpu(), want, atol=2e-5, rtol=1e-5)
        torch.testing.assert_close(state[slots[e]].cpu(), rows[-1], atol=2e-5, rtol=1e-5)
        base += n
    # final read-out of chosen rows: the sum of the streams, nothing written back
    pick = torch.tensor([t - 1, 0, 5], dtype=torch.int32)
    hl = torch.zeros(3, width, device=device)
    H.hyper_step(d(x), None, d(y), dc, None, dn, hl, si, gather=d(pick))
    torch.testing.assert_close(hl.cpu(), O.dynamic_tanh(new.sum(0), norm.alpha, norm.w, norm.b)[pick.long()], atol=3e-5, rtol=1e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("heads,dim,vdim", [(2, 44, 56), (3, 20, 36), (1, 64, 10), (2, 128, 130), (1, 200, 33), (4, 100, 32), (2, 256, 140)])
@pytest.mark.parametrize("segment", [0, 32])
@pytest.mark.parametrize("split", [False, True])
def test_hgrn2_recurrence(device, heads, dim, vdim, segment, split):
    """``split`` rounds v only: with v exact in tf32 the tensor-core blocks are as good as the fp32 steps."""
    if device == "cpu" and (split or segment):
        pytest.skip("variants of the CUDA kernel")
    g = torch.Generator().manual_seed(dim)
    si, order, _ = step_of(CHUNKS, device)
    t, hd = si.num_tokens, heads * dim
    qfv = torch.randn(t, 2 * hd + heads * vdim, generator=g)
    bias, low = torch.randn(hd, generator=g) + 3, torch.rand(hd, generator=g) * 0.9
    low[::3] = 0
    qfv[:, 2 * hd:] = qfv[:, 2 * hd:].bfloat16()
    qfv[3, hd:2 * hd] = -60.0            # a gate that closes: the state is replaced, nothing overflows
    rows = H.state_rows(dim)
    start = torch.randn(len(order), heads, vdim, rows, generator=g)
    start[..., dim:] = 0
    state, out = start.to(device).clone(), torch.zeros(t, heads * vdim, device=device)
    H.hgrn2(qfv.to(device), bias.to(device), low.to(device), state, out, heads, dim, vdim, si, segment=segment, split=split)
    base, slots = 0, si.state_slot.cpu()
    for e, (a, n) in enumerate(order):
        z = qfv[base:base + n].double()
        q = (z[:, :hd] * torch.sigmoid(z[:, :hd])).view(n, heads, dim)
        f = (low + (1 - low) * torch.sigmoid(z[:, hd:2 * hd] + bias.double())).view(n, heads, dim)
        v = z[:, 2 * hd:].view(n, heads, vdim)
        S = start[slots[e], :, :, :dim].double().transpose(1, 2) if a > 0 else torch.zeros(heads, dim, vdim, dtype=torch.float64)
        want = []
        for i in range(n):
            S = f[i][:, :, None] * S + (1 - f[i])[:, :, None] * v[i][:, None, :]
            want.append((q[i][:, :, None] * S).sum(1).reshape(-1))
        scale = torch.stack(want).abs().max()
        assert (out[base:base + n].cpu().double() - torch.stack(want)).abs().max() < 2e-5 * scale
        assert (state[slots[e], :, :, :dim].cpu().double().transpose(1, 2) - S).abs().max() < 2e-5 * S.abs().max()
        base += n
    w = torch.rand(vdim, generator=g)
    normed = torch.zeros(t, heads * vdim, device=device)
    H.head_rmsnorm(out, w.to(device), 1e-5, normed, heads, vdim)
    want = O.root_mean_square_norm(out.cpu().view(t, heads, vdim), w, 1e-5).reshape(t, -1)
    torch.testing.assert_close(normed.cpu(), want, atol=1e-5, rtol=1e-5)


def latent_case(device, dtype, heads, rank, window, chunks, spike, splits=1, counters=None):
    """Latent attention over random pages; with ``spike`` one latent outshines all others at a chosen distance."""
    g = torch.Generator().manual_seed(heads * 1000 + rank)
    si, order, pages = step_of(chunks, device, page_seed=3)
    ld = rank + (-rank) % 8
    pool = torch.zeros(pages, 16, ld)
    table = si.page_table.cpu()
    q = torch.zeros(si.num_tokens * heads, ld)
    q[:, :rank] = torch.randn(si.num_tokens * heads, rank, generator=g)
    lat = []
    for e, (a, n) in enumerate(order):
        c = torch.randn(a + n, rank, generator=g) * 0.5
        if spike is not None:
            far = a + n - 1 - spike      # seen by the last row iff spike < window
            if far >= 0:
                c[far] = 2.0
        lat.append(c)
    if spike is not None:
        q[:, :rank] = 0.6 + 0.05 * q[:, :rank]
    q, lat = q.to(dtype).float(), [c.to(dtype).float() for c in lat]
    for e, c in enumerate(lat):
        for j in range(len(c)):
            pool[table[e, j // 16], j % 16, :rank] = c[j]
    out = torch.zeros(si.num_tokens * heads, ld, dtype=dtype, device=device)
    part_o = torch.empty(si.num_tokens * heads * splits * ld, device=device)
    part_ml = torch.empty(si.num_tokens * heads * splits * 2, device=device)
    H.latent_attention(q.to(dtype).to(device), out, pool.to(dtype).to(device), si, heads, rank, 0.37, window, splits, part_o, part_ml, counters)
    base = 0
    for e, (a, n) in enumerate(order):
        c = lat[e].double()
        i, j = torch.arange(a, a + n)[:, None], torch.arange(a + n)[None, :]
        seen = (j <= i) & ((i - j < window) if window > 0 else (j >= 0))
        for hd in range(heads):
            rows = q[base * heads + hd:(base + n) * heads:heads, :rank].double()
            s = (rows @ c.T * 0.37).masked_fill(~seen, float("-inf"))
            want = torch.softmax(s, -1) @ c
            got = out[base * heads + hd:(base + n) * heads:heads, :rank].cpu().double()
            assert (got - want).abs().max() < (0.03 if dtype == torch.bfloat16 else 2e-5), (e, hd)
        base += n


@pytest.mark.parametrize("where", [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=GPU),
                                   pytest.param(("cuda", torch.bfloat16), marks=GPU)])
@pytest.mark.parametrize("heads,rank,window", [(3, 56, 21), (1, 18, 1), (6, 64, 80), (16, 128, 0), (5, 192, 100), (2, 512, 40), (4, 24, 16)])
def test_latent_attention_window_edges(where, heads, rank, window):
    chunks = [(7, 1), (0, 1), (window + 40, 1), (30, 2), (0, 2), (5, 17), (130, 70), (0, 150)]
    latent_case(*where, heads, rank, window, chunks, None)
    for spike in ((window - 1, window) if window > 0 else (90,)):      # just inside and just outside; far away without a window
        latent_case(*where, heads, rank, window, chunks, spike)


@GPU
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,rank,window,splits", [(3, 56, 0, 4), (16, 128, 300, 3), (2, 512, 200, 8), (32, 256, 0, 5)])
def test_latent_decode_with_split_keys(dtype, heads, rank, window, splits):
    chunks = [(7, 1), (0, 1), (400, 1), (255, 1), (15, 1), (16, 1), (299, 1), (300, 1)]
    counters = torch.zeros(len(chunks) * -(-heads // 16), dtype=torch.int32, device="cuda")
    for c in (None, counters, counters):                  # merged by a second kernel, or by a row's last split (counters come back as zeros)
        latent_case("cuda", dtype, heads, rank, window, chunks, None, splits, c)
        latent_case("cuda", dtype, heads, rank, window, chunks, window if window else 380, splits, c)
    assert (counters == 0).all()


@pytest.mark.parametrize("device", DEVICES)
def test_latent_append_norms_and_places(device):
    g = torch.Generator().manual_seed(5)
    c = torch.randn(9, 40, generator=g)
    w, slots = torch.rand(36, generator=g) + 0.5, torch.tensor([5, 16, 17, -1, 31, 0, 47, 33, 2], dtype=torch.int32)
    pool = torch.zeros(3, 16, 40, device=device)
    H.latent_append(c.to(device), 0, w.to(device), 1e-3, slots.to(device), pool, 36)
    flat = pool.cpu().view(48, 40)
    want = O.root_mean_square_norm(c[:, :36], w, 1e-3)
    for r, s in enumerate(slots.tolist()):
        if s >= 0:
            torch.testing.assert_close(flat[s, :36], want[r], atol=1e-5, rtol=1e-5)
    assert (flat[:, 36:] == 0).all() and (flat[1] == 0).all()


@GPU
@pytest.mark.parametrize("m,n,k,batch", [(1, 8, 8, 3), (5, 56, 24, 5), (130, 128, 64, 8), (300, 72, 200, 2), (64, 512, 128, 32), (257, 40, 512, 4)])
def test_batched_products(m, n, k, batch):
    g = torch.Generator().manual_seed(m)
    a, w = torch.randn(m, batch * k, generator=g).bfloat16(), torch.randn(batch * n, k, generator=g).bfloat16()
    step = n + 8
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 5e-3)):
        out = torch.full((m, batch * step), 7.0, dtype=dt, device="cuda")
        H.linear_batched(a.to(dt).cuda(), w.to(dt).cuda(), out, batch, k, step)
        for z in range(batch):
            want = a[:, z * k:(z + 1) * k].double() @ w[z * n:(z + 1) * n].double().T
            got = out[:, z * step:z * step + n].cpu().double()
            assert (got - want).abs().max() < tol * want.abs().max()
            assert (out[:, z * step + n:(z + 1) * step] == 7.0).all()      # nothing past a problem's columns
    ops.check_status()


@pytest.mark.parametrize("where", [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=GPU),
                                   pytest.param(("cuda", torch.bfloat16), marks=GPU)])
def test_gated_linear_gelu(where):
    device, dt = where
    g = torch.Generator().manual_seed(8)
    for m, inter, k, half in ((3, 64, 40, 64), (200, 96, 72, 32), (70, 256, 128, 128)):
        a = torch.randn(m, k, generator=g).to(dt)
        gate, up = (torch.randn(inter, k, generator=g) * 3 / k ** 0.5).to(dt), (torch.randn(inter, k, generator=g) / k ** 0.5).to(dt)
        out = torch.zeros(m, inter, dtype=dt, device=device)
        H.gated_linear(a.to(device), ops.pack_gate_up(gate, up, half).to(device), half, "gelu_tanh", out, torch.zeros(m, 2 * inter, dtype=dt, device=device))
        want = O.gelu_tanh(a.double() @ gate.double().T) * (a.double() @ up.double().T)
        assert (out.cpu().double() - want).abs().max() < (1e-5 if dt == torch.float32 else 8e-3) * want.abs().max()


@GPU
def test_fp32_linear_is_not_reduced_precision():
    g = torch.Generator().manual_seed(1)
    a, w = torch.randn(50, 300, generator=g), torch.randn(70, 300, generator=g)
    out = torch.zeros(50, 70, device="cuda")
    H.linear(a.cuda(), w.cuda(), out)
    want = a.double() @ w.double().T
    assert (out.cpu().double() - want).abs().max() < 3e-6 * want.abs().max()


@GPU
def test_fp32_argmax_and_sampler():
    g = torch.Generator().manual_seed(2)
    logits = torch.randn(9, 333, generator=g)
    dev = logits.cuda()
    assert torch.equal(ops.argmax(dev).cpu().long(), logits.argmax(-1))
    p = lambda v: torch.full((9,), v, device="cuda")
    args = (p(0.8), torch.full((9,), 20, dtype=torch.int32, device="cuda"), p(0.9), p(0.0), torch.linspace(0.01, 0.99, 9).cuda())
    got = ops.sample(dev, *args).cpu()
    assert torch.equal(got, ops.reference.sample(logits, *[a.cpu() for a in args]).to(got.dtype))


# ------------------------------------------------------------------------------------------
# the whole model through the engine
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", ENGINES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_layers(models, name, where):
    cfg, tensors = models[name]
    ids = tokens_of(cfg, 150, 1)
    streams = []
    want = O.forward(cfg, tensors, ids, layers_out=streams)
    eng = make_engine(cfg, tensors, where)
    eng.model.capture = []
    got = replay_cuts(eng, ids, [len(ids)])
    assert_logits(got, want, where)
    assert len(eng.model.capture) == len(cfg["layers"])
    for mine, ref in zip(eng.model.capture, streams):
        err = (mine[:150].cpu().double() - ref).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt()
        assert err < (0.02 if where[1] == "bf16" else 1e-5)


@pytest.mark.parametrize("where", ENGINES)
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("cuts", [[1], [2], [3, 1, 5, 2], [16], [17, 31, 1, 1, 64], [100, 1]])
def test_portions(models, name, where, cuts):
    cfg, tensors = models[name]
    ids = tokens_of(cfg, 118, 2)
    got = replay_cuts(make_engine(cfg, tensors, where), ids, cuts)
    assert_logits(got, O.forward(cfg, tensors, ids), where)


@pytest.mark.parametrize("where", ENGINES)
def test_unequal_requests_reuse_pages_and_slots(models, where):
    """Four live requests at most, a pool that holds no more than they need: portions beside decoded tokens, requests that
    pause, pages and slots handed on to the next request; every logits row as if alone."""
    cfg, tensors = models["mixed"]
    lengths = [100, 1, 37, 64, 90, 2, 16, 55, 33, 80]
    ids = {f"r{i}": tokens_of(cfg, n, 30 + i) for i, n in enumerate(lengths)}
    want = {k: O.forward(cfg, tensors, v) for k, v in ids.items()}
    rng = np.random.default_rng(3)
    eng = make_engine(cfg, tensors, where, max_tokens=320)
    rep, waiting, live, rows = replay.Replayer(eng), list(ids), {}, {k: [] for k in ids}
    used_slots = set()
    while waiting or live:
        while waiting and len(live) < 4 and sum(-(-len(ids[k]) // 64) * 64 for k in [*live, waiting[0]]) <= 320:
            live[waiting.pop(0)] = 0
        entries, end = [], []
        for k in list(live):
            if rng.random() < 0.25 and len(live) > 1:
                continue                                  # left out of this step, goes on later
            n = min(int(rng.choice([1, 1, 2, 3, 7, 16, 30, 64])), len(ids[k]) - live[k])
            entries.append({"id": k, "tokens": ids[k][live[k]:live[k] + n], "want": list(range(n))})
            live[k] += n
            if live[k] == len(ids[k]):
                end.append(k)
                del live[k]
        out = rep.step(entries, end)
        nseq = eng.si.num_decode + eng.si.num_prefill_seqs
        used_slots |= set(eng.plan_np[eng.L.state_slot:eng.L.state_slot + nseq].tolist()) if entries else set()
        for e in entries:
            rows[e["id"]] += [out.pop(0) for _ in e["want"]]
    for k in ids:
        assert_logits(torch.stack(rows[k]), want[k], where)
    assert eng.core.num_free_pages == eng.num_pages and eng.core.num_free_state_slots == 4 and used_slots <= {0, 1, 2, 3}


@pytest.mark.parametrize("where", ENGINES)
def test_window_releases_pages(models, where):
    """Pages behind the widest window go back to the pool while a sequence runs; a long sequence needs no more than that."""
    cfg, tensors = models["mixed"]                        # windows 21, 9 and 50: the widest decides
    ids = tokens_of(cfg, 230, 5)
    eng = make_engine(cfg, tensors, where, max_tokens=112, max_seq_len=400)
    got = replay_cuts(eng, ids, [9, 1, 1, 14, 2])
    assert_logits(got, O.forward(cfg, tensors, ids), where)


@pytest.mark.parametrize("where", ENGINES[:2])
def test_far_key_and_window_edge_show_in_logits(models, where):
    """Prompts that differ in one token at distance window - 1 or window from the last, under sharpened attention (32-bit
    engine only: three such layers magnify bf16 rounding itself)."""
    cfg, tensors = models["attention"]
    tensors = dict(tensors)
    for i in range(3):
        tensors[f"l{i}.mix.q"] = tensors[f"l{i}.mix.q"] * 3
    window = cfg["layers"][0]["mixer"]["mask"]["size"]
    base = tokens_of(cfg, 140, 6)
    for gap in (window - 1, window):
        a, b = list(base), list(base)
        a[139 - gap], b[139 - gap] = 3, 4                 # two prompts that differ in one far token
        eng = make_engine(cfg, tensors, where)
        for ids in (a, b):
            want = O.forward(cfg, tensors, ids)
            assert_logits(replay_cuts(eng, ids, [50, 2, 60, 1]), want, where)


@GPU
def test_prompts_on_expanded_latents(models):
    """Prompts with and without a past, beside decoded tokens, on the expanded keys and values; short portions stay on the
    latents; the two agree."""
    cfg, tensors = models["wide"]
    eng = make_engine(cfg, tensors, ("cuda", "bf16"), max_tokens=768)
    ids = {k: tokens_of(cfg, 240, 90 + i) for i, k in enumerate("abc")}
    want = {k: O.forward(cfg, tensors, v) for k, v in ids.items()}
    rep, at, rows = replay.Replayer(eng), dict.fromkeys("abc", 0), {k: [] for k in "abc"}
    count = lambda: ops.launch_counts["latent_expand"]
    for portions, expanded in (({"a": 130}, True), ({"a": 1, "b": 140}, True), ({"a": 1, "b": 2, "c": 1}, False), ({"a": 108, "b": 98, "c": 120}, True),
                               ({"c": 119}, True)):
        c0 = count()
        out = rep.step([{"id": k, "tokens": ids[k][at[k]:at[k] + n], "want": list(range(n))} for k, n in portions.items()], [])
        assert (count() > c0) == expanded
        for k, n in portions.items():
            rows[k] += [out.pop(0) for _ in range(n)]
            at[k] += n
    for k in "abc":
        assert_logits(torch.stack(rows[k]), want[k], ("cuda", "bf16"))


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
    # long decoding, far past every window
    r = eng.generate(prompts[0], GenerateOptions(max_new_tokens=120, greedy=True, ignore_eos=True))
    assert len(r.token_ids) == 120 and O.follows_greedily(cfg, tensors, prompts[0], r.token_ids)
    # a session continues (its history is computed again: there is no prefix to attach to)
    s = eng.create_session()
    first = eng.generate_in_session(s, prompts[4], GenerateOptions(max_new_tokens=3, greedy=True, ignore_eos=True))
    more = eng.generate_in_session(s, [7, 8], GenerateOptions(max_new_tokens=3, greedy=True, ignore_eos=True))
    assert O.follows_greedily(cfg, tensors, prompts[4] + first.token_ids + [7, 8], more.token_ids)


@pytest.mark.parametrize("device", DEVICES)
def test_preemption_recomputes_state(models, device):
    """A pool too small for all requests: victims lose pages and slot and are computed again, with the same tokens out."""
    cfg, tensors = models["attention"]
    eng = make_engine(cfg, tensors, (device, "f32"), max_tokens=224, max_seqs=4, num_pages=14, max_tokens_per_step=64, prefill_chunk=64, max_logit_rows=0)
    prompts = [tokens_of(cfg, n, 70 + n) for n in (40, 50, 45)]
    outs = eng.generate(prompts, max_new_tokens=40, ignore_eos=True)
    assert eng.core.num_preemptions > 0
    for p, o in zip(prompts, outs):
        assert len(o) == 40 and O.follows_greedily(cfg, tensors, p, o)


@pytest.mark.parametrize("device", DEVICES)
def test_forced_beside_generation(models, device):
    """Forced sequences and sampled requests share steps."""
    cfg, tensors = models["odd"]
    eng = make_engine(cfg, tensors, (device, "f32"))
    ids, prompt = tokens_of(cfg, 40, 8), tokens_of(cfg, 12, 9)
    want = O.forward(cfg, tensors, ids)
    sid = eng.add_request(prompt, 10, ignore_eos=True)
    fid = eng.open_forced(ids[:15], [0, 14])
    out, rows, at = [], {}, 15
    while len(out) < 10:
        step = eng.step()
        rows.update(step.forced_logits and {p: r.cpu() for p, r in step.forced_logits.get(fid, [])} or {})
        out += [t for s, t, _ in step.events if s == sid]
        if at < 40:
            eng.extend_forced(fid, ids[at:at + 5], [4])
            at += 5
    assert O.follows_greedily(cfg, tensors, prompt, out)
    assert set(rows) == {0, 14, 19, 24, 29, 34, 39}
    assert_logits(torch.stack([rows[p] for p in sorted(rows)]), want[sorted(rows)], (device, "f32"))
    assert not eng.has_work                               # an idle forced sequence is no work
    eng.close_forced(fid)
    with pytest.raises(ValueError, match="not an open forced"):
        eng.extend_forced(fid, [1])


def test_rewind_and_fork_start_over(models):
    cfg, tensors = models["recurrent"]
    eng = make_engine(cfg, tensors, ("cpu", "f32"), max_logit_rows=0)
    prompt = tokens_of(cfg, 20, 11)
    sid = eng.add_request(prompt, 30, ignore_eos=True)
    got = [t for _ in range(6) for s, t, _ in eng.step().events]
    assert eng.core.rewind(sid, 22) and eng.core.seq_computed(sid) == 0
    again = [t for _ in range(4) for s, t, _ in eng.step().events]
    assert len(again) == 4 and O.follows_greedily(cfg, tensors, prompt + got[:2], again)
    fid = eng.core.fork(sid)
    assert eng.core.seq_computed(fid) == 0
    events = [e for _ in range(3) for e in eng.step().events]
    assert [t for s, t, _ in events if s == fid][:2] == [t for s, t, _ in events if s == sid][:2]
    assert not eng.core.set_draft(sid, [1, 2])


def test_state_slots_bound_admission():
    core = Core(CoreConfig(num_pages=64, max_seqs=8, max_tokens_per_step=64, max_pages_per_seq=16, num_state_slots=2))
    plan = np.zeros(core.layout.total_words, dtype=np.int32)
    ids = [core.add_request([1, 2, 3], 5) for _ in range(3)]
    core.build_step(plan.ctypes.data)
    L = core.layout
    assert plan[2] == 2 and sorted(plan[L.state_slot:L.state_slot + 2].tolist()) == [0, 1] and core.num_waiting == 1
    core.commit_step(np.array([1, 1], dtype=np.int32).ctypes.data, 2)
    core.release(ids[0])
    core.build_step(plan.ctypes.data)
    assert core.num_waiting == 0 and plan[L.state_slot] != plan[L.state_slot + 1]


def test_what_state_rules_out_is_refused(models, tmp_path):
    cfg, tensors = models["odd"]
    for kw, what in (({"max_draft_tokens": 2}, "speculative"), ({"num_host_pages": 8}, "swap"), ({"kv_dtype": "fp8"}, "fp8")):
        with pytest.raises(ValueError, match=what):
            make_engine(cfg, tensors, ("cpu", "f32"), **{"compute_dtype": "bf16", **kw})
    bad = json.loads(json.dumps(cfg))
    bad["layers"][2]["mixer"]["kv_from"] = 1
    with pytest.raises(ValueError, match="kv_from"):
        registry.ARCHITECTURES["Rilelorn"].read_config(bad)
    c = registry.ARCHITECTURES["Rilelorn"].read_config(cfg)
    load = registry.ARCHITECTURES["Rilelorn"].load_weights
    assert load(c, {**tensors, "l9.extra": torch.zeros(1)}, torch.float32, "cpu").unused == ["l9.extra"]
    with pytest.raises(KeyError, match="l0.shift"):
        load(c, {k: v for k, v in tensors.items() if k != "l0.shift"}, torch.float32, "cpu")


def test_directory_commands_and_replay(models, tmp_path, capsys):
    from onnx_genai_b200 import cli

    cfg, tensors = models["odd"]
    d = write_checkpoint(tmp_path / "m", cfg, tensors)
    f = SafetensorsFile(d + "/model.safetensors")
    assert set(f) == set(tensors) and all(torch.equal(f[k], v) for k, v in tensors.items())
    assert cli.main(["show", d]) == 0
    assert json.loads(capsys.readouterr().out)["architecture"]["name"] == "Rilelorn"
    assert cli.main(["validate", d]) == 0 and json.loads(capsys.readouterr().out)["ok"]
    assert cli.main(["list", "--models-dir", str(tmp_path)]) == 0 and "m" in capsys.readouterr().out.split()
    prompt = tokens_of(cfg, 9, 4)
    rc = cli.main(["generate", d, "--device", "cpu", "--prompt-ids", ",".join(map(str, prompt)), "--greedy", "--max-new-tokens", "5"])
    out = [int(t) for t in capsys.readouterr().out.split()]
    assert rc == 0 and len(out) == 5 and O.follows_greedily(cfg, tensors, prompt, out)
    assert cli.main(["generate", d, "--device", "cpu", "--prompt", "text"]) == 2
    ids = tokens_of(cfg, 30, 5)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:20], "want": [3, 19]}, {"id": "b", "tokens": [1], "want": []}], "end": ["b"]},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[20:25], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": ids[25:], "want": [4]}], "end": ["a"]}]
    (tmp_path / "out").mkdir()
    said = []
    replay.serve(replay.build_engine(d, "float32", 128, "cpu"), str(tmp_path / "out"), io.StringIO("\n".join(map(json.dumps, lines))), said.append)
    assert said == ["done 0", "done 1", "done 2"] and sorted(p.name for p in (tmp_path / "out").iterdir()) == ["0.f32", "2.f32"]
    want = O.forward(cfg, tensors, ids)
    got = np.concatenate([np.fromfile(tmp_path / "out" / f"{s}.f32", dtype="<f4").reshape(-1, cfg["vocab"]) for s in (0, 2)])
    assert_logits(torch.from_numpy(got), want[[3, 19, 29]], ("cpu", "f32"))
