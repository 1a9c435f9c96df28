"""Slow, plain statement of the Fizesun decoder for the tests: torch on the CPU, one sequence, the whole sequence at once, one
function per mechanism.  It shares no code with the product path."""
import math

import torch


def rms(x, gain, eps):
    """x over its root mean square, times a gain (one number or one per coordinate)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


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


def rotate_pairs(x, dims, base, start=0):
    """x [n, d] at positions start, start + 1, ...: neighbours 2i, 2i + 1 of the first ``dims`` turn by position * base^(-2i / dims)."""
    out = x.clone()
    p = torch.arange(start, start + x.shape[0], dtype=torch.float64)
    for i in range(dims // 2):
        a = p * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        u, v = x[:, 2 * i], x[:, 2 * i + 1]
        out[:, 2 * i], out[:, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def latent(h, W, rank, eps):
    """(normed latents [n, rank], rotated key part before its rotation [n, rest])."""
    down = h @ W["dkv"].T
    return rms(down[:, :rank], W["dkv.norm"], eps), down[:, rank:]


def latent_attention(h, W, m, eps):
    n, H, d, r, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = latent(h, W, m["kv_rank"], eps)
    kr = rotate_pairs(kr, m["rot"]["dims"], m["rot"]["base"])
    q = (h @ W["q"].T).view(n, H, d + r)
    k, v = (c @ W["uk"].T).view(n, H, d), (c @ W["uv"].T).view(n, H, dv)
    i = torch.arange(n)
    seen = i[None, :] <= i[:, None]
    gate = sigmoid(h @ W["g"].T)
    heads = []
    for a in range(H):
        qr = rotate_pairs(q[:, a, d:], m["rot"]["dims"], m["rot"]["base"])
        s = (q[:, a, :d] @ k[:, a].T + qr @ kr.T) * m["scale"]
        s = s.masked_fill(~seen, float("-inf"))
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        heads.append((p / p.sum(-1, keepdim=True)) @ v[:, a] * gate[:, a:a + 1])
    return torch.cat(heads, -1) @ W["o"].T


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def xielu(z, p, q):
    rising = softplus(p) * z * z + z / 2
    falling = (0.5 + softplus(q)) * (torch.expm1(z.clamp(max=0)) - z) + z / 2
    return torch.where(z > 0, rising, falling)


def dense(h, W):
    return xielu(h @ W["up"].T, W["act"][0], W["act"][1]) @ W["down"].T


def limited_expert(h, gate, up, down, limit):
    g = (h @ gate.T).clamp(max=limit)
    u = (h @ up.T).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ down.T


def choose(logits, top):
    """Logits of one token -> (expert ids, weights): the largest, weighted by a softmax among themselves."""
    ids = sorted(range(len(logits)), key=lambda e: -float(logits[e]))[:top]
    z = torch.stack([logits[e] for e in ids])
    w = torch.exp(z - z.max())
    return ids, w / w.sum()


def experts(h, W, f):
    z = h @ W["router"].T + W["router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(*choose(z[t], f["router"]["top"])):
            out[t] += w * limited_expert(h[t], W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"], f["expert"]["limit"])
    if f.get("shared"):
        out += sigmoid(h @ W["shared.sg"].T) * limited_expert(h, W["shared.gate"], W["shared.up"], W["shared.down"], f["shared"]["limit"])
    return out


def enter_pass(x, x0, w_in, step):
    """What stands ahead of a pass through the looped layers."""
    return torch.cat([x, x0], -1) @ w_in.T + step


def layer_runs(cfg):
    """[(layer, number of the pass if one begins here, else None)] in the order they run."""
    loop, n, runs = cfg.get("loop"), len(cfg["layers"]), []
    if not loop:
        return [(i, None) for i in range(n)]
    runs += [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, tensors, ids, layers_out=None, dtype=torch.float64):
    """Logits [n, vocab] of one sequence; ``layers_out`` collects the residual stream after every layer run."""
    W = {k: v.to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x0 = x = rms(W["embed"][torch.as_tensor(ids, dtype=torch.long)], W["embed.norm"], eps)
    for i, begins in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        part = lambda kind: {k[len(p + kind):]: v for k, v in W.items() if k.startswith(p + kind)}
        if begins is not None:
            x = enter_pass(x, x0, W["loop.in"], W["loop.step"][begins])
        x = x + latent_attention(sublayer_input(rms(x, W[p + "norm1"], eps), W[p + "canon1"]), part("mix."), layer["mixer"], eps)
        f = layer["mlp"]
        if f is not None:
            h = sublayer_input(rms(x, W[p + "norm2"], eps), W[p + "canon2"])
            x = x + (dense(h, part("mlp.")) if f["kind"] == "dense" else experts(h, part("mlp."), f))
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms(x, W["final.norm"], eps) @ W["head"].T


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


def ff_experts(count, top, ff, limit=2.5, shared=None, shared_limit=1.25):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": count, "top": top},
            **({"shared": {"ff": shared, "limit": shared_limit}} if shared else {})}


def layer(heads, dim, rot_dim, vdim, rank, mlp, scale=None, base=700.0):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale or (dim + rot_dim) ** -0.5,
                      "rot": {"base": base, "dims": rot_dim}}}


def make_config(vocab, width, layers, loop=None, taps=3, eps=1e-4):
    """``loop``: (start, stop, times)."""
    return {"architecture": "Fizesun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "canon": {"taps": taps},
            **({"loop": dict(zip(("start", "stop", "times"), loop))} if loop else {})}


def random_tensors(cfg, seed=0, sharp=1.5):
    """bf16 weights; queries are scaled so that attention is far from uniform."""
    g = torch.Generator().manual_seed(seed)
    t, w = {}, cfg["width"]
    lin = lambda o, i, s=1.0: torch.randn(o, i, generator=g) * s / i ** 0.5
    one = lambda: 0.7 + 0.6 * torch.rand((), generator=g)
    t["embed"], t["embed.norm"] = torch.randn(cfg["vocab"], w, generator=g) * 0.3, one()
    if cfg.get("loop"):
        t["loop.in"], t["loop.step"] = lin(w, 2 * w), 0.4 * torch.randn(cfg["loop"]["times"], w, generator=g)
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        x, H = p + "mix.", m["heads"]
        t[p + "norm1"], t[p + "canon1"] = one(), torch.randn(w, cfg["canon"]["taps"], generator=g) * 0.4
        t[x + "q"], t[x + "dkv"] = lin(H * (m["dim"] + m["rot_dim"]), w, sharp), lin(m["kv_rank"] + m["rot_dim"], w)
        t[x + "dkv.norm"] = 0.6 + 0.8 * torch.rand(m["kv_rank"], generator=g)
        t[x + "uk"], t[x + "uv"] = lin(H * m["dim"], m["kv_rank"]), lin(H * m["vdim"], m["kv_rank"], 1.3)
        t[x + "g"], t[x + "o"] = lin(H, w, 1.5), lin(w, H * m["vdim"], 1.3)
        if f is None:
            continue
        t[p + "norm2"], t[p + "canon2"] = one(), torch.randn(w, cfg["canon"]["taps"], generator=g) * 0.4
        y = p + "mlp."
        if f["kind"] == "dense":
            t[y + "up"], t[y + "down"], t[y + "act"] = lin(f["ff"], w, 1.5), lin(w, f["ff"], 0.7), torch.randn(2, generator=g)
            continue
        n, ff = f["router"]["experts"], f["expert"]["ff"]
        t[y + "router"], t[y + "router.b"] = lin(n, w, 1.5), torch.randn(n, generator=g)
        for e in range(n):
            t[y + f"e{e}.gate"], t[y + f"e{e}.up"], t[y + f"e{e}.down"] = lin(ff, w, 2.0), lin(ff, w, 2.0), lin(w, ff)
        if f.get("shared"):
            ff = f["shared"]["ff"]
            t[y + "shared.gate"], t[y + "shared.up"], t[y + "shared.down"], t[y + "shared.sg"] = lin(ff, w, 2.0), lin(ff, w, 2.0), lin(w, ff), lin(1, w)
    t["final.norm"], t["head"] = one(), lin(cfg["vocab"], w, 2.0)
    return {k: v.bfloat16() for k, v in t.items()}
