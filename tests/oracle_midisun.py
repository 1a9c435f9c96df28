"""Slow, plain statement of the Midisun decoder for the tests: torch on the CPU, one sequence, the whole sequence at once, one
function per mechanism.  It shares no code with the product path."""

import torch


def rms(x, gain, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def rms_in_groups(x, gain, groups, eps):
    """Every one of ``groups`` equal consecutive parts over its own root mean square, then the gain."""
    part = x.shape[-1] // groups
    out = []
    for g in range(groups):
        y = x[..., g * part:(g + 1) * part]
        out.append(y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps))
    return torch.cat(out, -1) * gain


def causal_filter(h, w):
    """h [n, channels], w [channels, taps]: the last tap meets the token itself, earlier ones what came before (zeros at the start)."""
    n, taps = h.shape[0], w.shape[1]
    rows = []
    for t in range(n):
        acc = torch.zeros_like(h[0])
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                acc = acc + w[:, j] * h[s]
        rows.append(acc)
    return torch.stack(rows)


def sublayer_input(h, w):
    return h + causal_filter(h, w)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return torch.where(z > 0, -torch.log1p(torch.exp(-z.abs())), z - torch.log1p(torch.exp(-z.abs())))


def residual_gate(h, w, b):
    return sigmoid(h @ w.T + b)


def rotate_halves(x, dims, base, start=0):
    """x [n, d] at positions start, start + 1, ...: dimension i turns with i + dims / 2 by position * base^(-2i / dims)."""
    out = x.clone()
    p = torch.arange(start, start + x.shape[0], dtype=torch.float64)
    for i in range(dims // 2):
        a = p * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        u, v = x[:, i], x[:, i + dims // 2]
        out[:, i], out[:, i + dims // 2] = u * c - v * s, v * c + u * s
    return out


# ------------------------------------------------------------------------------------------
# mixers
# ------------------------------------------------------------------------------------------
def slope(a, heads):
    return 2.0 ** (-8.0 * (a + 1) / heads)


def attention_head(q, k, v, scale, cap, bias, window, sink):
    """One head over one sequence: capped scores, a bias that grows with the distance, a window and a sink in the denominator."""
    n = q.shape[0]
    i = torch.arange(n)
    dist = i[:, None] - i[None, :]
    s = q @ k.T * scale
    s = cap * torch.tanh(s / cap)
    s = s - bias * dist.to(s.dtype)
    s = s.masked_fill((dist < 0) | (dist >= window), float("-inf"))
    top = torch.maximum(s.max(-1, keepdim=True).values, sink)
    p = torch.exp(s - top)
    return (p @ v) / (p.sum(-1, keepdim=True) + torch.exp(sink - top))


def attention(h, W, m, eps):
    n, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ W["q"].T + W["q.b"], h @ W["k"].T + W["k.b"]
    v = k.view(n, G, d)
    q, k = rms(q, W["q.norm"], eps).view(n, H, d), rms(k, W["k.norm"], eps).view(n, G, d)
    gate = sigmoid(h @ W["g"].T)
    heads = []
    for a in range(H):
        g = a // (H // G)
        o = attention_head(q[:, a], k[:, g], v[:, g], m["scale"], m["softcap"], slope(a, H), m["mask"]["size"], W["sink"][a])
        heads.append(o * gate[:, a:a + 1])
    return torch.cat(heads, -1) @ W["o"].T + W["o.b"]


def retention_head(q, k, v, decay):
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    rows = []
    for t in range(q.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        rows.append(S.T @ q[t])
    return torch.stack(rows)


def retention(h, W, m, eps):
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ W[x].T).view(n, H, -1) for x in "qkv")
    heads = []
    for a in range(H):
        qa = rotate_halves(q[:, a], m["rot"]["dims"], m["rot"]["base"])
        ka = rotate_halves(k[:, a], m["rot"]["dims"], m["rot"]["base"]) * d ** -0.5
        heads.append(rms(retention_head(qa, ka, v[:, a], m["decay"][a]), 1.0, eps))
    return (torch.cat(heads, -1) * silu(h @ W["g"].T)) @ W["o"].T


def matrix_memory_head(q, k, v, i, f):
    """i, f [n]: log gates of the input and of the memory."""
    S, norm = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype), torch.zeros(q.shape[1], dtype=q.dtype)
    m = torch.zeros((), dtype=q.dtype)
    rows = []
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S, norm, m = keep * S + take * torch.outer(k[t], v[t]), keep * norm + take * k[t], new
        rows.append((S.T @ q[t]) / (torch.maximum((norm @ q[t]).abs(), torch.exp(-m)) + 1e-6))
    return torch.stack(rows)


def memory_gates(h, W, cap):
    capped = lambda z: cap * torch.tanh(z / cap)
    return capped(h @ W["i"].T + W["i.b"]), log_sigmoid(capped(h @ W["f"].T + W["f.b"]))


def matrix_memory(h, W, m, eps):
    n, H, d = h.shape[0], m["heads"], m["dim"]
    q, k, v = ((h @ W[x].T).view(n, H, -1) for x in "qkv")
    i, f = memory_gates(h, W, m["gate_cap"])
    heads = [rms(matrix_memory_head(q[:, a] * d ** -0.5, k[:, a], v[:, a], i[:, a], f[:, a]), 1.0, eps) for a in range(H)]
    return (torch.cat(heads, -1) * W["norm"] * sigmoid(h @ W["g"].T)) @ W["o"].T


MIXERS = {"attention": attention, "retention": retention, "mlstm": matrix_memory}


# ------------------------------------------------------------------------------------------
# feed-forwards
# ------------------------------------------------------------------------------------------
def gated(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def choose(z, correction, top, groups=1, keep=1):
    """Router logits of one token -> (expert ids, weights): chosen by corrected scores among the best groups, weighted without the correction."""
    s = sigmoid(z)
    c = s + correction
    per = len(z) // groups
    worth = lambda g: float(sum(sorted(c[g * per:(g + 1) * per].tolist())[-2:]))
    kept = sorted(range(groups), key=lambda g: -worth(g))[:keep]
    ids = sorted((e for e in range(len(z)) if e // per in kept), key=lambda e: -float(c[e]))[:top]
    w = torch.stack([s[e] for e in ids])
    return ids, w / (w.sum() + 1e-20)


def experts(h, W, f):
    r = f["router"]
    z = h @ W["router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, w = choose(z[t], W["correction"], r["top"], r["groups"]["count"], r["groups"]["keep"])
        for e, share in zip(ids, w):
            out[t] += share * gated(h[t], W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"])
    return out


def forward(cfg, tensors, ids, layers_out=None, dtype=torch.float64):
    """Logits [n, vocab] of one sequence; ``layers_out`` collects the residual stream after every layer."""
    W = {k: v.to(dtype) for k, v in tensors.items()}
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = W["embed"][torch.as_tensor(ids, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        part = lambda kind: {k[len(p + kind):]: v for k, v in W.items() if k.startswith(p + kind)}
        h = rms_in_groups(x, W[p + "norm1"], groups, eps)
        y = MIXERS[layer["type"]](sublayer_input(h, W[p + "canon1"]), part("mix."), layer["mixer"], eps)
        x = x + y * residual_gate(h, W[p + "rg1"], W[p + "rg1.b"])
        f = layer["mlp"]
        if f is not None:
            h = rms_in_groups(x, W[p + "norm2"], groups, eps)
            W2 = part("mlp.")
            y = gated(h, W2["gate"], W2["up"], W2["down"]) if f["kind"] == "dense" else experts(h, W2, f)
            x = x + y * residual_gate(h, W[p + "rg2"], W[p + "rg2.b"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_in_groups(x, W["final.norm"], groups, eps) @ W["head"].T


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
def ff_dense(ff):
    return {"kind": "dense", "ff": ff}


def ff_experts(count, top, ff, groups=1, keep=1):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": count, "top": top, "groups": {"count": groups, "keep": keep}}}


def attention_layer(heads, kv_heads, dim, window, mlp, scale=None, softcap=30.0):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "softcap": softcap,
                                                       "scale": scale or dim ** -0.5, "mask": {"size": window}}}


def retention_layer(heads, dim, vdim, mlp, decay=None, rot=None, base=900.0):
    """``decay``: the heads' (default: spread between fast and slow)."""
    decay = decay or [1 - 2.0 ** -(3 + 1.5 * a) for a in range(heads)]
    return {"type": "retention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay,
                                                       "rot": {"base": base, "dims": dim if rot is None else rot}}}


def memory_layer(heads, dim, vdim, mlp, cap=12.0):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def make_config(vocab, width, layers, groups=2, taps=3, eps=1e-4, scale=0.8):
    return {"architecture": "Midisun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps, "groups": groups}, "canon": {"taps": taps},
            "embedding": {"scale": scale}}


def random_tensors(cfg, seed=0, sharp=1.5):
    """bf16 weights; gates, sinks and corrections are far from where they would not show."""
    g = torch.Generator().manual_seed(seed)
    t, w = {}, cfg["width"]
    rnd = lambda *s: torch.randn(*s, generator=g)
    lin = lambda o, i, s=1.0: rnd(o, i) * s / i ** 0.5
    gain = lambda n: 0.6 + 0.8 * torch.rand(n, generator=g)
    t["embed"] = rnd(cfg["vocab"], w)
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        x, H = p + "mix.", m["heads"]
        t[p + "norm1"], t[p + "canon1"] = gain(w), rnd(w, cfg["canon"]["taps"]) * 0.4
        t[p + "rg1"], t[p + "rg1.b"] = lin(w, w, 1.5), rnd(w)
        kv = m["kv_heads"] * m["dim"] if layer["type"] == "attention" else H * m["dim"]
        out = H * m["vdim"]
        t[x + "q"], t[x + "k"], t[x + "o"] = lin(H * m["dim"], w, sharp), lin(kv, w, sharp), lin(w, out, 1.3)
        if layer["type"] == "attention":
            t[x + "q.b"], t[x + "k.b"], t[x + "o.b"] = rnd(H * m["dim"]) * 0.5, rnd(kv) * 0.5, rnd(w) * 0.3
            t[x + "q.norm"], t[x + "k.norm"] = sharp * gain(H * m["dim"]), gain(kv)
            t[x + "sink"], t[x + "g"] = 1 + rnd(H), lin(H, w, 1.5)
        else:
            t[x + "v"], t[x + "g"] = lin(out, w), lin(out, w, 1.5)
        if layer["type"] == "mlstm":
            t[x + "norm"] = gain(out)
            t[x + "i"], t[x + "i.b"], t[x + "f"], t[x + "f.b"] = lin(H, w, 3.0), rnd(H), lin(H, w, 3.0), 2 + rnd(H)
        if f is None:
            continue
        t[p + "norm2"], t[p + "rg2"], t[p + "rg2.b"] = gain(w), lin(w, w, 1.5), rnd(w)
        y = p + "mlp."
        if f["kind"] == "dense":
            t[y + "gate"], t[y + "up"], t[y + "down"] = lin(f["ff"], w, 1.5), lin(f["ff"], w, 1.5), lin(w, f["ff"])
            continue
        n, ff = f["router"]["experts"], f["expert"]["ff"]
        t[y + "router"], t[y + "correction"] = lin(n, w, 1.5), rnd(n) * 0.5
        for e in range(n):
            t[y + f"e{e}.gate"], t[y + f"e{e}.up"], t[y + f"e{e}.down"] = lin(ff, w, 2.0), lin(ff, w, 2.0), lin(w, ff)
    t["final.norm"], t["head"] = gain(w), lin(cfg["vocab"], w, 2.0)
    return {k: v.bfloat16() for k, v in t.items()}
