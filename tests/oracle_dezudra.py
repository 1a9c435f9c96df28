"""Slow, plain statement of the Dezudra decoder for the tests: torch on the CPU, one sequence, the whole sequence at once, one
function per mechanism.  It shares no code with the product path."""
import math

import torch


def rms_norm(x, w, eps):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z / (1 + torch.exp(-z))


def causal_conv(u, w):
    """u [n, channels], w [channels, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    n, taps = u.shape[0], w.shape[1]
    rows = []
    for t in range(n):
        acc = torch.zeros_like(u[0])
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                acc = acc + w[:, j] * u[s]
        rows.append(acc)
    return torch.stack(rows)


def rotate(x, dims, base):
    """x [n, dim] at positions 0 .. n - 1: dimension i turns with dimension i + dims / 2; the rest passes."""
    n, half = x.shape[0], dims // 2
    out = x.clone()
    for i in range(half):
        a = torch.arange(n, dtype=torch.float64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        u, v = x[:, i], x[:, i + half]
        out[:, i], out[:, i + half] = u * c - v * s, v * c + u * s
    return out


def visible(n, window, keep):
    """seen[i, j]: query i sees key j (window 0: every earlier token)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    return seen & ((i - j < window) | (j < keep)) if window > 0 else seen


def softmax_attention(q, k, v, scale, seen):
    s = ((q @ k.T) * scale).masked_fill(~seen, float("-inf"))
    p = torch.exp(s - s.max(-1, keepdim=True).values)
    return (p / p.sum(-1, keepdim=True)) @ v


def mix_lambda(W, diff):
    return torch.exp((W["lq1"] * W["lk1"]).sum()) - torch.exp((W["lq2"] * W["lk2"]).sum()) + diff


def differential_attention(h, W, m, eps):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = causal_conv(h @ W["q"].T + W["q.b"], W["q.conv"]).view(n, H, 2, d)
    k = causal_conv(h @ W["k"].T + W["k.b"], W["k.conv"]).view(n, G, 2, d)
    v = causal_conv(h @ W["v"].T + W["v.b"], W["v.conv"]).view(n, G, dv)
    seen = visible(n, m["mask"]["size"], m["mask"]["keep_first"])
    lam = mix_lambda(W, m["diff"])
    heads = []
    for a in range(H):
        g = a // (H // G)
        maps = []
        for i in range(2):
            qr, kr = rotate(q[:, a, i], m["rot"]["dims"], m["rot"]["base"]), rotate(k[:, g, i], m["rot"]["dims"], m["rot"]["base"])
            maps.append(softmax_attention(qr, kr, v[:, g], m["scale"], seen))
        heads.append(rms_norm(maps[0] - lam * maps[1], None, eps) * (1 - m["diff"]))
    return torch.cat(heads, -1) @ W["o"].T


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def log_decay(z, A_log):
    """log of the decay for z = W_a h + dt_bias."""
    return -torch.exp(A_log) * torch.where(z > 20, z, torch.log1p(torch.exp(z.clamp(max=20))))


def delta_rule(q, k, v, decay, beta):
    """One head, token after token: q, k [n, d], v [n, dv], decay, beta [n] -> o [n, dv]."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype)
    rows = []
    for t in range(q.shape[0]):
        S = decay[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        rows.append(S.T @ q[t])
    return torch.stack(rows)


def gated_delta(h, W, m, eps):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit(silu(causal_conv(h @ W["q"].T, W["q.conv"])).view(n, G, d)) * d ** -0.5
    k = unit(silu(causal_conv(h @ W["k"].T, W["k.conv"])).view(n, G, d))
    v = silu(causal_conv(h @ W["v"].T, W["v.conv"])).view(n, H, dv)
    beta = 1 / (1 + torch.exp(-(h @ W["b"].T)))
    decay = torch.exp(log_decay(h @ W["a"].T + W["dt_bias"], W["A_log"]))
    gate = silu(h @ W["g"].T).view(n, H, dv)
    heads = []
    for a in range(H):
        g = a // (H // G)
        o = delta_rule(q[:, g], k[:, g], v[:, a], decay[:, a], beta[:, a])
        heads.append(rms_norm(o, W["norm"], eps) * gate[:, a])
    return torch.cat(heads, -1) @ W["o"].T


def choose_experts(scores, top, count, keep):
    """scores [experts] of one token -> chosen expert ids: the best of the ``keep`` best of ``count`` groups of neighbours."""
    size = len(scores) // count
    best = sorted(range(count), key=lambda g: -max(scores[g * size:(g + 1) * size].tolist()))[:keep]
    allowed = [e for g in best for e in range(g * size, (g + 1) * size)]
    return sorted(allowed, key=lambda e: -float(scores[e]))[:top]


def experts_forward(h, W, m):
    """Squared-relu experts, weighted by their softmax scores as they are."""
    r = m["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    scores = torch.softmax(h @ W["router"].T, -1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose_experts(scores[t], r["top"], groups["count"], groups["keep"]):
            a = (W[f"e{e}.up"] @ h[t]).clamp(min=0)
            out[t] += scores[t, e] * (W[f"e{e}.down"] @ (a * a))
    return out


def forward(cfg, tensors, ids, layers_out=None, dtype=torch.float64):
    """Logits [n, vocab] of one sequence; ``layers_out`` collects the residual stream after every layer."""
    W = {k: v.to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(ids)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        part = lambda kind: {k[len(p + kind):]: v for k, v in W.items() if k.startswith(p + kind)}
        mixer = {"attention": differential_attention, "delta": gated_delta}[layer["type"]]
        y = mixer(rms_norm(x, W[p + "norm1"], eps), part("mix."), layer["mixer"], eps)
        x = x + rms_norm(y, W[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            y = experts_forward(rms_norm(x, W[p + "norm2"], eps), part("mlp."), layer["mlp"])
            x = x + rms_norm(y, W[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T * cfg["logit_scale"]


def follows_greedily(cfg, tensors, prompt, generated, slack=2e-4):
    """Every generated token is (up to ``slack``) the best continuation of what came before it."""
    logits = forward(cfg, tensors, list(prompt) + list(generated))
    for i, tok in enumerate(generated):
        row = logits[len(prompt) - 1 + i]
        if row.max() - row[tok] > slack * row.std():
            return False
    return True


# ------------------------------------------------------------------------------------------
# configurations and weights for the tests
# ------------------------------------------------------------------------------------------
def experts(count, top, ff, groups=1, keep=1):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": count, "top": top, "groups": {"count": groups, "keep": keep}}}


def layer_attention(heads, kv_heads, dim, vdim, window, keep, mlp, conv=3, rot=None, base=1000.0, diff=0.4, scale=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "diff": diff,
                      "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": window, "keep_first": keep},
                      "rot": {"base": base, "dims": dim if rot is None else rot}}}


def layer_delta(heads, kv_heads, dim, vdim, mlp, conv=4):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def make_config(vocab, width, layers, eps=1e-5, logit_scale=1.5):
    return {"architecture": "Dezudra", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "logit_scale": logit_scale}


def random_tensors(cfg, seed=0, sharp=2.0):
    """bf16 weights; queries and keys are scaled so that attention is far from uniform."""
    g = torch.Generator().manual_seed(seed)
    t = {}
    lin = lambda o, i, s=1.0: torch.randn(o, i, generator=g) * s / i ** 0.5
    near = lambda n, spread=0.3: 1 + spread * (torch.rand(n, generator=g) - 0.5)
    w = cfg["width"]
    t["embed"] = torch.randn(cfg["vocab"], w, generator=g)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        taps = lambda n: torch.randn(n, m["conv"], generator=g) * 0.5 / m["conv"] ** 0.5 + torch.eye(m["conv"])[-1]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] else ()):
            t[p + n] = near(w)
        x = p + "mix."
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            for n, rows, s in (("q", 2 * H * d, sharp), ("k", 2 * G * d, 1.0), ("v", G * dv, 1.0)):
                t[x + n], t[x + n + ".b"], t[x + n + ".conv"] = lin(rows, w, s), 0.3 * torch.randn(rows, generator=g), taps(rows)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                t[x + n] = torch.randn(d, generator=g) * 0.35 / d ** 0.25
        else:
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                t[x + n], t[x + n + ".conv"] = lin(rows, w, 1.5), taps(rows)
            t[x + "b"], t[x + "a"], t[x + "g"] = lin(H, w), lin(H, w), lin(H * dv, w)
            t[x + "A_log"], t[x + "dt_bias"] = torch.rand(H, generator=g) * 2 - 2, torch.randn(H, generator=g) - 2
            t[x + "norm"] = near(dv)
        t[x + "o"] = lin(w, H * dv)
        if layer["mlp"]:
            y, n, ff = p + "mlp.", layer["mlp"]["router"]["experts"], layer["mlp"]["expert"]["ff"]
            t[y + "router"] = lin(n, w, 1.5)
            for e in range(n):
                t[y + f"e{e}.up"], t[y + f"e{e}.down"] = lin(ff, w), lin(w, ff)
    t["final.norm"], t["head"] = near(w), lin(cfg["vocab"], w, 2.0)
    return {k: v.bfloat16() for k, v in t.items()}
