"""Slow, plain statement of the Rilelorn decoder for the tests: float64 or float32 torch on the CPU, one sequence, the whole
sequence at once, one function per mechanism.  It shares no code with the product path."""
import math

import torch


def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def root_mean_square_norm(x, w, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


def token_shift(h, amount):
    """Every row moves towards the row before it; zeros stand before the first."""
    before = torch.zeros_like(h)
    before[1:] = h[:-1]
    return h + (before - h) * amount


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def read_streams(streams, weight):
    """streams [s, n, width] -> the weighted sum a sublayer reads."""
    out = torch.zeros_like(streams[0])
    for k in range(streams.shape[0]):
        out = out + weight[k] * streams[k]
    return out


def write_streams(streams, mix, out_weight, y):
    new = []
    for t in range(streams.shape[0]):
        acc = out_weight[t] * y
        for s in range(streams.shape[0]):
            acc = acc + mix[s, t] * streams[s]
        new.append(acc)
    return torch.stack(new)


def hgrn2(h, W, heads, dim, vdim, eps):
    """h [n, width]; W: q f f.b lower v norm o.  One token after the other."""
    n = h.shape[0]
    z = h @ W["q"].T
    q = (z * torch.sigmoid(z)).view(n, heads, dim)
    v = (h @ W["v"].T).view(n, heads, vdim)
    low = W["lower"]
    f = (low + (1 - low) * torch.sigmoid(h @ W["f"].T + W["f.b"])).view(n, heads, dim)
    S = torch.zeros(heads, dim, vdim, dtype=h.dtype)
    rows = []
    for t in range(n):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        o = (q[t][:, :, None] * S).sum(1)
        rows.append(root_mean_square_norm(o, W["norm"], eps).reshape(-1))
    return torch.stack(rows) @ W["o"].T


def latent(h, W, eps):
    return root_mean_square_norm(h @ W["dkv"].T, W["dkv.norm"], eps)


def latent_attention(h, c, W, heads, dim, vdim, scale, window):
    """h [n, width] queries; c [n, rank] latents; keys and values are expanded head by head."""
    n = h.shape[0]
    q = (h @ W["q"].T).view(n, heads, dim)
    k = (c @ W["uk"].T).view(n, heads, dim)
    v = (c @ W["uv"].T).view(n, heads, vdim)
    i = torch.arange(n)
    gap = i[:, None] - i[None, :]
    seen = (gap >= 0) & (gap < window)
    out = []
    for a in range(heads):
        s = (q[:, a] @ k[:, a].T) * scale
        s = s.masked_fill(~seen, float("-inf"))
        out.append(torch.softmax(s, -1) @ v[:, a])
    return torch.cat(out, -1) @ W["o"].T


def gated_mlp(h, gate, up, down):
    return (gelu_tanh(h @ gate.T) * (h @ up.T)) @ down.T


def forward(config, tensors, tokens, dtype=torch.float64, layers_out=None):
    """Logits [n, vocab] of one sequence.  ``tensors``: name -> tensor; ``layers_out``: list that gets the summed streams
    after every layer."""
    T = {k: v.to(dtype) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = T["embed"][tokens].repeat(config["streams"], 1, 1)

    def norm(name, u):
        return dynamic_tanh(u, T[name + ".alpha"], T[name], T[name + ".b"])

    latents = {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        W = {k[len(p) + 4:]: v for k, v in T.items() if k.startswith(p + "mix.")}
        h = token_shift(norm(p + "norm1", read_streams(x, T[p + "hc1.in"])), T[p + "shift"])
        if layer["type"] == "hgrn2":
            y = hgrn2(h, W, m["heads"], m["dim"], m["vdim"], eps)
        else:
            src = m.get("kv_from")
            if src is None:
                latents[i] = latent(h, W, eps)
            y = latent_attention(h, latents[i if src is None else src], W, m["heads"], m["dim"], m["vdim"], m["scale"], m["mask"]["size"])
        x = write_streams(x, T[p + "hc1.mix"], T[p + "hc1.out"], y)
        if layer["mlp"] is not None:
            h = norm(p + "norm2", read_streams(x, T[p + "hc2.in"]))
            y = gated_mlp(h, T[p + "mlp.gate"], T[p + "mlp.up"], T[p + "mlp.down"])
            x = write_streams(x, T[p + "hc2.mix"], T[p + "hc2.out"], y)
        if layers_out is not None:
            layers_out.append(x.sum(0))
    return norm("final.norm", x.sum(0)) @ T["head"].T


# ------------------------------------------------------------------------------------------
# small random checkpoints
# ------------------------------------------------------------------------------------------
def layer_hgrn2(heads, dim, vdim, ff):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def layer_latent(heads, dim, vdim, rank, window, ff, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale or dim ** -0.5, "mask": {"size": window}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def make_config(vocab, width, streams, layers, eps=1e-5):
    return {"architecture": "Rilelorn", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "layers": layers}


def random_tensors(config, seed=0):
    g = torch.Generator().manual_seed(seed)
    W, S = config["width"], config["streams"]
    out = {}

    def normal(name, *shape, gain=1.0):
        out[name] = (torch.randn(*shape, generator=g) * gain / shape[-1] ** 0.5).to(torch.bfloat16)

    def uniform(name, *shape, lo=0.0, hi=1.0):
        out[name] = (lo + (hi - lo) * torch.rand(*shape, generator=g)).to(torch.bfloat16)

    def norm(name):
        uniform(name, W, lo=0.6, hi=1.4)
        uniform(name + ".b", W, lo=-0.3, hi=0.3)
        uniform(name + ".alpha", 1, lo=0.5, hi=1.1)
        out[name + ".alpha"] = out[name + ".alpha"].reshape(())

    def hyper(name):
        uniform(name + ".in", S, lo=0.2, hi=1.2)
        uniform(name + ".out", S, lo=-0.4, hi=1.2)
        uniform(name + ".mix", S, S, lo=-0.2, hi=0.4)
        out[name + ".mix"] += torch.eye(S, dtype=torch.bfloat16) * 0.5

    normal("embed", config["vocab"], W, gain=W ** 0.5)
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        norm(p + "norm1")
        uniform(p + "shift", W, lo=0.1, hi=0.9)
        hyper(p + "hc1")
        if layer["type"] == "hgrn2":
            hd, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            normal(p + "mix.q", hd, W, gain=1.5)
            normal(p + "mix.f", hd, W, gain=2.0)
            uniform(p + "mix.f.b", hd, lo=0.0, hi=4.0)
            uniform(p + "mix.lower", hd, lo=0.0, hi=0.9)
            normal(p + "mix.v", hv, W, gain=1.5)
            uniform(p + "mix.norm", m["vdim"], lo=0.5, hi=1.5)
            normal(p + "mix.o", W, hv, gain=1.5)
        else:
            normal(p + "mix.q", m["heads"] * m["dim"], W, gain=2.5)
            if "kv_from" not in m:
                normal(p + "mix.dkv", m["kv_rank"], W)
                uniform(p + "mix.dkv.norm", m["kv_rank"], lo=0.5, hi=1.5)
            normal(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"], gain=2.5)
            normal(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"], gain=1.5)
            normal(p + "mix.o", W, m["heads"] * m["vdim"], gain=1.5)
        if layer["mlp"]:
            norm(p + "norm2")
            hyper(p + "hc2")
            ff = layer["mlp"]["ff"]
            normal(p + "mlp.gate", ff, W, gain=1.5)
            normal(p + "mlp.up", ff, W)
            normal(p + "mlp.down", W, ff, gain=1.5)
    norm("final.norm")
    normal("head", config["vocab"], W, gain=2.0)
    return out


def follows_greedily(config, tensors, prompt, out):
    """True when every token of ``out`` is the most likely one after what precedes it."""
    logits = forward(config, tensors, list(prompt) + list(out)[:-1])
    return logits[len(prompt) - 1:].argmax(-1).tolist() == list(out)
