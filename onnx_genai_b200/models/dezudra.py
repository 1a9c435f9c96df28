"""Dezudra: differential-attention and gated-delta layers behind short convolutions, squared-relu experts, one residual stream with
RMS norms before and behind every sublayer.

Reads a checkpoint directory's ``config.json`` and ``model.safetensors`` into the generic hybrid configuration and weights
(models/hybrid.py).  Every size and constant comes from the configuration or a tensor's shape.
"""
from __future__ import annotations

import math

from .hybrid import (DeltaSpec, DiffSpec, HybridConfig, HybridLayer, HybridWeights, LayerSpec, MoeSpec, pack_delta, pack_diff, pack_moe, pad_cols)
from ..ops.hybrid import RmsNorm


def read_config(doc: dict, name: str = "dezudra") -> HybridConfig:
    layers = []
    for i, entry in enumerate(doc["layers"]):
        m, mlp = entry["mixer"], entry.get("mlp")
        sizes = dict(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), taps=int(m["conv"]))
        if entry["type"] == "delta":
            mixer = DeltaSpec(**sizes)
        elif entry["type"] == "attention":
            mask, rot = m.get("mask") or {}, m.get("rot") or {}
            mixer = DiffSpec(**sizes, scale=float(m["scale"]), diff=float(m["diff"]), window=int(mask.get("size", 0)), keep=int(mask.get("keep_first", 0)),
                             rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 1.0)))
        else:
            raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
        ff = None
        if mlp is not None:
            if mlp["kind"] != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            r = mlp["router"]
            groups = r.get("groups") or {"count": 1, "keep": 1}
            ff = MoeSpec(experts=int(r["experts"]), top=int(r["top"]), inter=int(mlp["expert"]["ff"]), groups=int(groups["count"]), keep=int(groups["keep"]))
        layers.append(LayerSpec(mixer, ff))
    cfg = HybridConfig(vocab=int(doc["vocab"]), hidden=int(doc["width"]), layers=layers, norm_eps=float(doc["norm"]["eps"]), name=name, residual="sandwich",
                       logit_scale=float(doc.get("logit_scale", 1.0)))
    cfg.validate()
    return cfg


def load_weights(cfg: HybridConfig, tensors, dtype, device) -> HybridWeights:
    """``tensors``: name -> CPU tensor mapping (package/safetensors.py reads the file)."""
    used = set()

    def take(name, f32=False):
        used.add(name)
        t = tensors[name].to(device)
        return t.float() if f32 else t.to(dtype)

    def norm(name, scale=1.0):
        return RmsNorm((take(name, True) * scale).contiguous(), cfg.norm_eps)

    w = HybridWeights(embed=take("embed"))
    for i, spec in enumerate(cfg.layers):
        p, m = f"l{i}.", spec.mixer
        x = lambda name, f32=False: take(p + "mix." + name, f32)
        three = lambda end: [x(n + end, True) for n in "qkv"]
        if isinstance(m, DeltaSpec):
            mixer = pack_delta(m, x("q"), x("k"), x("v"), x("g"), x("a"), x("b"), three(".conv"), x("A_log", True), x("dt_bias", True), x("norm", True), x("o"))
        else:
            dot = [float((x("lq" + n, True).double() * x("lk" + n, True).double()).sum()) for n in "12"]
            mixer = pack_diff(m, x("q"), x("k"), x("v"), three(".b"), three(".conv"), math.exp(dot[0]) - math.exp(dot[1]) + m.diff, x("o"))
        layer = HybridLayer(norm1=norm(p + "norm1"), hc1=norm(p + "norm1b"), mixer=mixer)
        if spec.mlp is not None:
            layer.norm2, layer.hc2 = norm(p + "norm2"), norm(p + "norm2b")
            e = range(spec.mlp.experts)
            layer.moe = pack_moe(take(p + "mlp.router"), [take(f"{p}mlp.e{k}.up") for k in e], [take(f"{p}mlp.e{k}.down") for k in e])
        w.layers.append(layer)
    w.final_norm, w.lm_head = norm("final.norm", cfg.logit_scale), pad_cols(take("head"))     # the scale of the logits rides in the last norm
    w.unused = sorted(set(tensors) - used)
    return w
