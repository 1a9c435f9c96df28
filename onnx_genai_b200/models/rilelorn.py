"""Rilelorn: HGRN2 and latent-attention layers on hyper-connected streams with Dynamic-Tanh norms and token shift.

Reads a checkpoint directory's ``config.json`` and ``model.safetensors`` into the generic hybrid configuration and weights
(models/hybrid.py).  Every size and constant comes from the configuration or a tensor's shape.
"""
from __future__ import annotations

from .hybrid import (HybridConfig, HybridLayer, HybridWeights, LatentSpec, LayerSpec, MlpSpec, RecurrentSpec, pack_latent, pack_mlp,
                     pack_recurrent, pad_cols)
from ..ops.hybrid import DynamicTanh, HyperConnection


def read_config(doc: dict, name: str = "rilelorn") -> HybridConfig:
    layers = []
    for i, entry in enumerate(doc["layers"]):
        m, mlp = entry["mixer"], entry.get("mlp")
        if entry["type"] == "hgrn2":
            mixer = RecurrentSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]))
        elif entry["type"] == "latent_attention":
            mask = m.get("mask")
            src = m.get("kv_from")
            mixer = LatentSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), rank=int(m["kv_rank"]), scale=float(m["scale"]),
                               window=int(mask["size"]) if mask else 0, kv_from=None if src is None else int(src))
        else:
            raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        layers.append(LayerSpec(mixer, MlpSpec(int(mlp["ff"])) if mlp is not None else None))
    cfg = HybridConfig(vocab=int(doc["vocab"]), hidden=int(doc["width"]), layers=layers, streams=int(doc.get("streams", 1)),
                       norm_eps=float(doc["norm"]["eps"]), name=name)
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
        return DynamicTanh(take(name + ".alpha", True).reshape(1), take(name, True), take(name + ".b", True))

    def conn(name):
        return HyperConnection(read=take(name + ".in", True), write=take(name + ".out", True), mix=take(name + ".mix", True).contiguous())

    w = HybridWeights(embed=take("embed"))
    for i, spec in enumerate(cfg.layers):
        p, m = f"l{i}.", spec.mixer
        x = lambda name, f32=False: take(p + "mix." + name, f32)
        if isinstance(m, RecurrentSpec):
            mixer = pack_recurrent(m, x("q"), x("f"), x("f.b", True), x("lower", True), x("v"), x("norm", True), x("o"))
        else:
            own = m.kv_from is None
            mixer = pack_latent(m, x("q"), x("dkv") if own else None, x("dkv.norm", True) if own else None, x("uk"), x("uv"), x("o"))
        layer = HybridLayer(norm1=norm(p + "norm1"), shift=take(p + "shift", True), hc1=conn(p + "hc1"), mixer=mixer)
        if spec.mlp is not None:
            layer.norm2, layer.hc2 = norm(p + "norm2"), conn(p + "hc2")
            pack_mlp(layer, take(p + "mlp.gate"), take(p + "mlp.up"), take(p + "mlp.down"))
        w.layers.append(layer)
    w.final_norm, w.lm_head = norm("final.norm"), pad_cols(take("head"))
    w.unused = sorted(set(tensors) - used)
    return w
