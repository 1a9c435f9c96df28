"""Midisun: attention over keys that are the values (norm over the whole projection, soft cap, distance bias, window, sink, head gates),
retention and mLSTM layers behind input convolutions; dense silu and sigmoid-routed expert feed-forwards; one residual stream with an RMS
norm in groups before every sublayer and a gate on what the sublayer adds.

Reads a checkpoint directory's ``config.json`` and ``model.safetensors`` into the generic hybrid configuration and weights
(models/hybrid.py).  Every size and constant comes from the configuration or a tensor's shape.
"""
from __future__ import annotations

import torch

from .hybrid import (HybridConfig, HybridLayer, HybridWeights, LayerSpec, MemorySpec, MlpSpec, MoeSpec, TiedSpec, distance_slopes, pack_gated_moe,
                     pack_input_conv, pack_memory, pack_mlp, pack_tied, pad_cols)
from ..ops.hybrid import RmsNorm


def read_mixer(i: int, kind: str, m: dict):
    if kind == "attention":
        if int(m.get("vdim", m["dim"])) != int(m["dim"]):
            raise ValueError(f"layer {i}: values of {m['vdim']} for keys of {m['dim']}; they are the keys in this design")
        return TiedSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0),
                        window=int((m.get("mask") or {}).get("size", 0)))
    sizes = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]))
    if kind == "retention":
        rot = m.get("rot") or {}
        return MemorySpec(**sizes, decay=tuple(map(float, m["decay"])), rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 1.0)))
    if kind == "mlstm":
        return MemorySpec(**sizes, gate_cap=float(m["gate_cap"]))
    raise ValueError(f"layer {i}: unknown mixer type {kind!r}")


def read_mlp(i: int, mlp: dict | None):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return MlpSpec(int(mlp["ff"]), "silu")
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    return MoeSpec(experts=int(r["experts"]), top=int(r["top"]), inter=int(mlp["expert"]["ff"]), groups=int(groups["count"]), keep=int(groups["keep"]),
                   group_best=2, score="sigmoid", renormalize=True, act="silu", bias=True)


def read_config(doc: dict, name: str = "midisun") -> HybridConfig:
    layers = [LayerSpec(read_mixer(i, entry["type"], entry["mixer"]), read_mlp(i, entry.get("mlp"))) for i, entry in enumerate(doc["layers"])]
    cfg = HybridConfig(vocab=int(doc["vocab"]), hidden=int(doc["width"]), layers=layers, norm_eps=float(doc["norm"]["eps"]), name=name, residual="pre",
                       norm_groups=int(doc["norm"].get("groups", 1)), input_taps=int(doc["canon"]["taps"]), ff_input_conv=False, residual_gates=True,
                       embed_scale=float((doc.get("embedding") or {}).get("scale", 1.0)), embed_normed=False)
    cfg.validate()
    return cfg


def load_weights(cfg: HybridConfig, tensors, dtype, device) -> HybridWeights:
    """``tensors``: name -> CPU tensor mapping (package/safetensors.py reads the file)."""
    used = set()

    def take(name, f32=False):
        used.add(name)
        t = tensors[name].to(device)
        return t.float() if f32 else t.to(dtype)

    def norm(name):
        return RmsNorm(take(name, True).contiguous(), cfg.norm_eps, cfg.norm_groups)

    w = HybridWeights(embed=take("embed"))
    for i, spec in enumerate(cfg.layers):
        p, m, f = f"l{i}.", spec.mixer, spec.mlp
        x = lambda name, f32=False: take(p + "mix." + name, f32)
        if isinstance(m, TiedSpec):
            mixer = pack_tied(m, x("q"), x("k"), x("g"), x("q.b", True), x("k.b", True), x("q.norm", True), x("k.norm", True),
                              distance_slopes(m.heads, device), x("sink", True), x("o"), x("o.b", True))
        else:
            own = dict(gates=torch.cat([x("i"), x("f")], 0), gates_bias=torch.cat([x("i.b", True), x("f.b", True)]), norm=x("norm", True)) if m.gated else {}
            mixer = pack_memory(m, x("q"), x("k"), x("v"), x("g"), x("o"), **own)
        layer = HybridLayer(norm1=norm(p + "norm1"), hc1=None, mixer=mixer, conv1=pack_input_conv(take(p + "canon1", True)), gate1=pad_cols(take(p + "rg1")),
                            gate1_bias=take(p + "rg1.b", True).contiguous())
        if f is not None:
            layer.norm2, layer.gate2, layer.gate2_bias = norm(p + "norm2"), pad_cols(take(p + "rg2")), take(p + "rg2.b", True).contiguous()
        y = lambda name, f32=False: take(p + "mlp." + name, f32)
        if isinstance(f, MoeSpec):
            part = lambda kind: [y(f"e{e}.{kind}") for e in range(f.experts)]
            layer.moe = pack_gated_moe(y("router"), y("correction", True), part("gate"), part("up"), part("down"))
        elif f is not None:
            pack_mlp(layer, y("gate"), y("up"), y("down"), f.act)
        w.layers.append(layer)
    w.final_norm, w.lm_head = norm("final.norm"), pad_cols(take("head"))
    w.unused = sorted(set(tensors) - used)
    return w
